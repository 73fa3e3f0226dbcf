"""Prefill and decode throughput of a Gatarax-style model beside the closest models of equal size (a Redodra-style model:
the gated delta rule and a state space behind short convolutions, attention with forms of the score; a Lulisun-style model:
plain window attention, routed experts; a dense decoder), and the time of each of its kernels against its roofline
(`python bench.py --arch gatarax`).

All models get random bf16 weights and the same width, depth, heads and head size.  The Gatarax model has four layers:
window attention with a sink beside the delta rule with decays per key channel, with a dense feed-forward and with routed
experts, and two layers of fixed-decay linear attention, likewise.  A kernel's roofline time is the slowest of its
multiply-adds at the measured bf16 throughput, its bytes at the measured copy bandwidth and, for the recurrences and the
router, its float32 multiply-adds at the FFMA pipe's nominal rate; `x_roofline` is measured time over that.  Timed with CUDA
events after warm-up, a 256 MiB write between iterations (flushes L2).
"""
from __future__ import annotations

import json
import math
import sys
import time

import torch

from . import arch_bench, redodra_bench
from .arch_bench import Timer, _roofline_ms, _step_context, ffma_peak_tflops, throughput
from .vadodra_bench import dense_norm_and_rope

# the Redodra sizes (width, attention heads / kv heads / head size, window, heads of the delta rule, dense feed-forward, the
# Lulisun model's experts), and the taps in front of the sublayers, the short convolutions' taps and the low ranks
SIZES = {name: dict(s, taps=4, conv=4, rank=rank) for (name, s), rank in zip(redodra_bench.SIZES.items(), (64, 128, 128))}


def gatarax_config(s: dict) -> dict:
    hd = s["hd"]
    left = {"heads": s["heads"], "kv_heads": s["kv"], "dim": hd, "vdim": hd, "scale": 1.0 / math.sqrt(hd), "conv": s["conv"],
            "mask": {"size": s["window"]}}
    right = {"heads": s["dheads"], "kv_heads": s["dheads"], "dim": hd, "vdim": hd, "conv": s["conv"], "decay_rank": s["rank"],
             "gate_rank": s["rank"]}
    light = {"heads": s["dheads"], "dim": hd, "vdim": hd, "decay": [1.0 - 2.0 ** -(1 + 8 * h / s["dheads"]) for h in range(s["dheads"])]}
    dense = {"kind": "dense", "ff": s["ff"]}
    moe = {"kind": "moe", "expert": {"ff": s["eff"]},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": s["egroups"], "keep": s["ekeep"]}}}
    side = {"left": left, "right": right}
    return {"architecture": "Gatarax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "canon": {"taps": s["taps"]},
            "embedding": {"scale": 1.0}, "logit_scale": 1.0, "layers": [
                {"type": "parallel", "mixer": side, "mlp": dense}, {"type": "lightning", "mixer": light, "mlp": moe},
                {"type": "lightning", "mixer": light, "mlp": dense}, {"type": "parallel", "mixer": side, "mlp": moe}]}


def time_parts(engine, s: dict, lens_before: list, new_tokens: int, peaks: dict, timer: Timer) -> dict:
    """Milliseconds of the Gatarax model's mixers and feed-forwards and of their kernels alone, for a step of `new_tokens`
    tokens per sequence on top of `lens_before` cached positions, with each kernel's roofline."""
    from . import attention as attn_kernels, linear, ops, tcgen05
    slots, ctx = _step_context(engine, lens_before, new_tokens, s["vocab"], 5)
    dev, bf, f32 = engine.device, torch.bfloat16, torch.float32
    n, width, B = ctx.n_tokens, s["width"], len(lens_before)
    residual = torch.zeros(n, width, dtype=f32, device=dev)
    x = (torch.randn(n, width, device=dev) * 0.5).to(bf)
    out = {}

    def row(name, ms, flops, bytes_, fp32_flops=0.0):
        ideal = _roofline_ms(flops, bytes_, peaks, fp32_flops)
        times = {"tensor": flops / (peaks["bf16_tflops"] * 1e12), "hbm": bytes_ / (peaks["hbm_gbs"] * 1e9),
                 "ffma": fp32_flops / (peaks["fp32_ffma_tflops_nominal"] * 1e12)}
        out[name] = {"ms": round(ms, 4), "roofline_ms": round(ideal, 6), "x_roofline": round(ms / ideal, 2),
                     "bound": max(times, key=times.get)}

    blocks = [layer.block for layer in engine.model.layers]
    # ---- the norm with both input convolutions -------------------------------------------------------------------
    stream = torch.randn(n, width, device=dev)
    a, b = (torch.empty(n, width, dtype=bf, device=dev) for _ in range(2))
    blk, carried = blocks[0], engine.cache.layer(0).parts[1].state
    row("norm_and_input_convolutions", timer(lambda: blk.mixer_conv.run(stream, blk.norm, blk.mixer_conv, blk.feed_forward_conv, carried, a, b, ctx)),
        0.0, n * width * (4 + 2 + 2) + width * 4 * (1 + 2 * s["taps"]) + 2 * B * carried[0].numel() * 4)

    # ---- window attention (left member of layer 0) ---------------------------------------------------------------
    par, cache0 = blk.mixer, engine.cache.layer(0).parts[0]
    (_, left), (_, right) = par.members
    left_cache, right_cache = cache0.parts
    out["parallel_mixer_ms"] = round(timer(lambda: par.forward(x, residual, ctx, cache0, True)), 4)
    hd, heads, kv, window = s["hd"], s["heads"], s["kv"], s["window"]
    vis = kv_bytes = 0
    for before in lens_before:
        vis += sum(min(window, p + 1) for p in range(before, before + new_tokens))
        kv_bytes += (before + new_tokens - max(0, before - window + 1)) * kv * 2 * hd * 2
    keys, proj = left_cache.parts
    both = torch.zeros(n, par.w_in.n, device=dev)
    project = linear.accumulate_split if linear.wants_split(x, par.w_in) else linear.logits           # as the part calls it
    row("members_projection", timer(lambda: project(x, par.w_in, both, ctx)), 2.0 * n * par.w_in.n * width,
        par.w_in.n * width * 2 + n * (width * 2 + par.w_in.n * 4))
    z = torch.randn(n, left.w_qkv.n, device=dev) * 0.5
    q = torch.empty(n, left.q_dim, dtype=bf, device=dev)
    ms = timer(lambda: ops.conv_store(z, left.b_qkv, left.w_conv, proj.state, q, keys.k, keys.v, ctx.cu_seqlens, ctx.token_pos,
                                      ctx.token_seq, ctx.seq_slot, ctx.page_table, n_seqs=ctx.n_seqs, n_kv_heads=kv, head_dim=hd,
                                      v_head_dim=hd, page_size=ctx.page_size, longest_run=ctx.max_new))
    row("convolve_store", ms, 0.0, n * left.w_qkv.n * 6 + left.w_qkv.n * 4 * (1 + s["conv"]) + 2 * B * proj.state[0].numel() * 4)
    mixed = torch.empty(n, left.o_dim, dtype=bf, device=dev)
    ms = timer(lambda: attn_kernels.attention(q, keys, mixed, ctx, n_heads=heads, n_kv_heads=kv, head_dim=hd, scale=left.scale,
                                              window=window, sink=left.sinks))
    row("window_attention", ms, 4.0 * hd * vis * heads, kv_bytes + n * heads * hd * 2 * 2)
    joined = [(torch.randn(n, width, device=dev), bias, w, 0.5) for w, bias in zip(par.norm_weights, (left.b_o, None))]
    row("normed_sum", timer(lambda: ops.normed_sum(joined, residual, 1e-5, accumulate=True, clear=both if project is linear.accumulate_split else None)), 0.0, n * width * (2 * 8 + 8))

    # ---- the delta rule with decays per key channel (right member) ----------------------------------------------------
    matrix, conv = right_cache.parts
    H, G, dim, vdim = right.n_heads, right.n_kv_heads, right.head_dim, right.v_head_dim
    z = torch.randn(n, right.width, device=dev) * 0.5
    u = torch.empty(n, -(-(right.conv_ch + 2 * H) // 4) * 4, dtype=f32, device=dev)
    decay = torch.empty(n, H * dim, dtype=f32, device=dev)
    gate = torch.empty(n, right.v_dim, dtype=f32, device=dev)
    common = dict(conv_col=0, conv_ch=right.conv_ch, taps=right.w_conv, conv_state=conv.state, unit_heads=2 * G, unit_dim=dim,
                  scaled_heads=G, unit_scale=dim ** -0.5, heads=H, step_col=right.beta_col, a_log=right.a_log, dt_bias=right.dt_bias,
                  out=u, cu_seqlens=ctx.cu_seqlens, token_seq=ctx.token_seq, seq_slot=ctx.seq_slot, n_seqs=ctx.n_seqs,
                  longest_run=ctx.max_new)
    # convolved channels read and written, the low-rank inputs read, decays and gates written, the maps read once
    maps = s["rank"] * (H * dim + right.v_dim)
    row("delta_prepare", timer(lambda: right._prepare_channels(z, 0, decay, gate, n, ctx, common)), 2.0 * n * maps,
        n * (right.conv_ch * 8 + (H * dim + right.v_dim) * 4 + 2 * s["rank"] * 4 + H * 8) + maps * 2 + 2 * B * conv.state[0].numel() * 4)
    o = torch.empty(n, right.v_dim, dtype=f32, device=dev)
    ms = timer(lambda: ops.state_scan(u, matrix.state, o, ctx.cu_seqlens, ctx.seq_slot, n_seqs=ctx.n_seqs, heads=H, groups=G, dim=dim,
                                      vdim=vdim, q_col=0, k_col=right.qk_dim, v_col=2 * right.qk_dim, decay_col=0,
                                      step_col=right.conv_ch + H, delta=True, decay=decay, longest_run=ctx.max_new))
    row("delta_scan", ms, 0.0, n * (H * (3 * dim + vdim + 1) + H * vdim) * 4 + 2 * B * H * dim * vdim * 4, fp32_flops=8.0 * n * H * dim * vdim)
    normed = torch.empty(n, right.v_dim, dtype=bf, device=dev)
    ms = timer(lambda: ops.gated_group_norm(o, gate, 0, right.norm, normed, groups=H, group_size=vdim, gate_first=False,
                                            gate_act="sigmoid", eps=1e-5))
    row("delta_gated_norm", ms, 0.0, n * H * vdim * (4 + 4 + 2))

    # ---- fixed-decay linear attention (layer 1) --------------------------------------------------------------------
    lt, cache1 = blocks[1].mixer, engine.cache.layer(1).parts[0]
    out["lightning_mixer_ms"] = round(timer(lambda: lt.forward(x, residual, ctx, cache1, True)), 4)
    H, dim, vdim = lt.n_heads, lt.head_dim, lt.v_head_dim
    z = torch.randn(n, lt.width, device=dev) * 0.5
    row("lightning_projection", timer(lambda: linear.logits(x, lt.w_in, z, ctx, silu_cols=lt.activated)), 2.0 * n * lt.width * width,
        lt.width * width * 2 + n * (width * 2 + lt.width * 4))
    o = torch.empty(n, lt.v_dim, dtype=f32, device=dev)
    row("lightning_scan", timer(lambda: lt.scan(z, cache1, o, ctx)), 0.0,
        n * (H * (2 * dim + vdim) + H * vdim) * 4 + 2 * B * H * dim * vdim * 4, fp32_flops=6.0 * n * H * dim * vdim)
    normed = torch.empty(n, lt.v_dim, dtype=bf, device=dev)
    ms = timer(lambda: ops.gated_group_norm(o, z, lt.gate_col, lt.norm, normed, groups=1, group_size=lt.v_dim, gate_first=False,
                                            gate_act="sigmoid", eps=1e-5))
    row("lightning_gated_norm", ms, 0.0, n * lt.v_dim * (4 + 4 + 2))

    # ---- feed-forwards ---------------------------------------------------------------------------------------------
    ff = blocks[0].feed_forward
    out["dense_feed_forward_ms"] = round(timer(lambda: ff.forward(x, residual, ctx)), 4)
    inter = ff.intermediate_size
    act = torch.empty(n, inter, dtype=bf, device=dev)
    row("up_activation", timer(lambda: linear.activated(x, ff.w_up, act, ctx, ff.act)), 2.0 * n * inter * width,
        inter * width * 2 + n * (width + inter) * 2)
    row("down", timer(lambda: linear.into_residual(act, ff.w_down, residual, ctx)), 2.0 * n * inter * width,
        inter * width * 2 + n * (inter * 2 + width * 8))
    mx = blocks[1].feed_forward
    out["experts_feed_forward_ms"] = round(timer(lambda: mx.forward(x, residual, ctx)), 4)
    top, experts, f = mx.top, mx.n_experts, mx.expert_size
    pairs = n * top
    ids = torch.empty(n, top, dtype=torch.int32, device=dev)
    wts = torch.empty(n, top, dtype=f32, device=dev)
    route = lambda: ops.moe_route(x, mx.router, None, ids, wts, top=top, groups=mx.n_groups, keep=mx.group_keep, softmax=True,
                                  normalise=False, group_max=True, **mx.route_cut(x, ctx))
    row("router", timer(route), 0.0, experts * width * 4 + n * width * 2, fp32_flops=2.0 * n * experts * width)
    used = int(torch.unique(ids).numel())
    if not mx._on_tensor_cores(x):
        raise RuntimeError("the benchmark's experts run on the tensor cores")
    rows = tcgen05.GROUPED_TILE_ROWS
    i32 = lambda k: torch.zeros(k, dtype=torch.int32, device=dev)
    offsets, order, tiles, n_tiles, place = i32(experts + 1), i32(pairs), i32(2 * (-(-pairs // rows) + experts)), i32(1), i32(pairs)
    arrange = lambda: ops.moe_arrange(ids, pairs, experts, rows, offsets, order, tiles, n_tiles, place)
    arrange()
    y = torch.empty(pairs, width, dtype=f32, device=dev)
    acts = torch.empty(pairs, f, dtype=bf, device=dev)
    xs = torch.zeros(pairs, width, dtype=bf, device=dev)
    gather = lambda: ops.moe_gather(x, xs, order, n_pairs=pairs, top=top)
    gather()
    ms_up = timer(lambda: tcgen05.grouped_gemm(xs, mx.w_gate, mx.w_up, acts, offsets, tiles, n_tiles, n_pairs=pairs))
    ms_down = timer(lambda: tcgen05.grouped_gemm(acts, mx.w_down, None, y, offsets, tiles, n_tiles, n_pairs=pairs))
    out["gather_ms"], out["arrange_ms"] = round(timer(gather), 4), round(timer(arrange), 4)
    row("experts_gate_up", ms_up, 2.0 * pairs * 2 * f * width, used * 2 * f * width * 2 + pairs * (width + f) * 2)
    row("experts_down", ms_down, 2.0 * pairs * f * width, used * f * width * 2 + pairs * (f * 2 + width * 4))
    row("combine", timer(lambda: ops.moe_combine(residual, y, wts, top=top, place=place)), 0.0, pairs * width * 4 + n * width * 8 + pairs * 8)
    out["experts_used"] = used
    engine.workspace.rezero()
    for slot in slots:
        engine.free_slot(slot)
    return out


# how far each kernel of the design is from its roofline, over the like kernel of the closest model
LIKE = {"norm_and_input_convolutions": ("dense", "rms_norm"), "window_attention": ("lulisun", "attention"),
        "convolve_store": ("dense", "rotate_store"), "members_projection": ("dense", "down"),
        "lightning_projection": ("dense", "down"), "normed_sum": ("redodra", "normed_sum"), "delta_prepare": ("redodra", "delta_rule_prepare"),
        "delta_scan": ("redodra", "delta_rule_scan"), "delta_gated_norm": ("redodra", "delta_rule_gated_norm"),
        "lightning_scan": ("redodra", "state_space_scan"), "lightning_gated_norm": ("redodra", "state_space_gated_norm"),
        "up_activation": ("redodra", "up_activation"), "down": ("dense", "down"), "experts_gate_up": ("lulisun", "experts_gate_up"),
        "experts_down": ("lulisun", "experts_down")}


def main(sizes: str, peaks: dict, peak_source: str, *, prefill_tokens: int = 2048, batch: int = 8, context: int | None = None,
         steps: int = 64) -> int:
    from ..config.registry import config_from_dict
    from ..engine.engine import Engine
    s = SIZES[sizes]
    if context is None:
        context = s["window"] + s["window"] // 4        # the window layers see a full window
    torch.cuda.set_device(0)
    timer = Timer("cuda:0")
    peaks = dict(peaks, fp32_ffma_tflops_nominal=round(ffma_peak_tflops(), 1))
    cache_tokens = batch * (context + steps + 128) + prefill_tokens + 4096
    result = {"arch": "gatarax", "sizes": sizes, "config": s, "dtype": "bf16", "data": "synthetic (random weights, random token ids)",
              "peaks": dict(peaks, source=peak_source), "l2": "256 MiB written between timed iterations"}
    ls = redodra_bench._lulisun_sizes(s)
    models = (("gatarax", gatarax_config(s)), ("redodra", redodra_bench.redodra_config(s)), ("lulisun", arch_bench.lulisun_config(ls)),
              ("dense", redodra_bench.dense_config(s, cache_tokens)))
    for kind, cfg in models:
        t0 = time.time()
        engine = Engine.from_random(config_from_dict(cfg), seed=0, std=0.02, dtype="bfloat16", device="cuda:0",
                                    max_tokens=cache_tokens, n_slots=batch + 2)
        print(f"[bench] {kind} ready in {time.time() - t0:.1f} s", file=sys.stderr, flush=True)
        r = throughput(engine, s, prefill_tokens=prefill_tokens, batch=batch, context=context, steps=steps, timer=timer)
        for phase, before, new in (("prefill_parts", [0], prefill_tokens), ("decode_parts", [context] * batch, 1)):
            if kind == "gatarax":
                r[phase] = time_parts(engine, s, before, new, peaks, timer)
            elif kind == "redodra":
                r[phase] = redodra_bench.time_parts(engine, s, before, new, peaks, timer)
            elif kind == "lulisun":
                r[phase] = arch_bench.time_parts(engine, "lulisun", ls, before, new, peaks, timer)
            else:
                r[phase] = arch_bench.time_parts(engine, "dense", s, before, new, peaks, timer)
                r[phase].update(dense_norm_and_rope(engine, s, before, new, peaks, timer))
        engine.check_device_status()
        result[kind] = r
        del engine
        torch.cuda.empty_cache()
    ratios = {}
    for phase in ("prefill_parts", "decode_parts"):
        for name, (model, other) in LIKE.items():
            ratios[f"{phase[:-6]}.{name} (over {model} {other})"] = round(
                result["gatarax"][phase][name]["x_roofline"] / result[model][phase][other]["x_roofline"], 2)
        for name, other in (("router", "route_ms"), ("combine", "combine_ms")):
            ratios[f"{phase[:-6]}.{name} ms (over lulisun {name} ms)"] = round(
                result["gatarax"][phase][name]["ms"] / max(result["lulisun"][phase][other], 1e-6), 2)
    result["x_roofline_over_like"] = ratios
    print(json.dumps(result))
    return 0
