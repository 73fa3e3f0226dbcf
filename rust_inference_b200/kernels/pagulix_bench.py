"""Prefill and decode throughput of a Pagulix-style model beside the closest models of equal size (a Vadodra-style model:
attention over a shared latent; a Redodra-style model: the gated delta rule; a Lulisun-style model: attention, routed
experts; a dense decoder), and the time of each of its kernels against its roofline (`python bench.py --arch pagulix`).

All models get random bf16 weights and the same width, depth, heads and head size.  The Pagulix model has four layers, each
with routed experts and a shared one: latent attention over a window with sinks, attention (values narrower than keys), the
delta rule, and attention whose values blend in the first one's.  A kernel's roofline time is the slowest of its multiply-adds at
the measured bf16 throughput, its bytes at the measured copy bandwidth and, for the recurrence and the router, its float32
multiply-adds at the FFMA pipe's nominal rate; `x_roofline` is measured time over that.  Timed with CUDA events after warm-up,
a 256 MiB write between iterations (flushes L2).
"""
from __future__ import annotations

import json
import math
import sys
import time

import torch

from . import arch_bench, redodra_bench, vadodra_bench
from .arch_bench import Timer, _roofline_ms, _step_context, ffma_peak_tflops, throughput
from .vadodra_bench import dense_norm_and_rope

# the Redodra sizes (width, attention heads / kv heads / head size, window, rotated channels, heads of the delta rule, the Lulisun
# model's experts), the Vadodra latent's, the streams and the attention's value heads
SIZES = {name: dict(s, streams=streams, vd=64, **{k: vadodra_bench.SIZES[name][k] for k in ("lheads", "ldim", "lrot", "lvdim", "rank")})
         for (name, s), streams in zip(redodra_bench.SIZES.items(), (2, 4, 2))}


def pagulix_config(s: dict) -> dict:
    lat = {"heads": s["lheads"], "dim": s["ldim"], "rot_dim": s["lrot"], "vdim": s["lvdim"], "kv_rank": s["rank"],
           "scale": 1.0 / math.sqrt(s["ldim"] + s["lrot"]), "rot": {"base": 10000.0, "dims": s["lrot"]}, "mask": {"size": s["window"]}}
    attn = {"heads": s["heads"], "kv_heads": s["kv"], "dim": s["hd"], "vdim": s["vd"], "scale": 1.0 / math.sqrt(s["hd"]), "v_mix": True,
            "rot": {"base": 500000.0, "dims": s["rot"], "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    delta = {"heads": s["dheads"], "kv_heads": s["dheads"], "dim": s["hd"], "vdim": s["hd"], "conv": 4}
    moe = {"kind": "moe", "expert": {"ff": s["eff"]}, "router": {"experts": s["experts"], "top": s["top"]}, "shared": {"ff": s["shared"]}}
    return {"architecture": "Pagulix", "vocab": s["vocab"], "width": s["width"], "streams": s["streams"], "residual_mult": 0.7,
            "logit_softcap": 30.0, "norm": {"eps": 1e-5}, "layers": [
                {"type": "latent_attention", "mixer": lat, "mlp": moe}, {"type": "attention", "mixer": attn, "mlp": moe},
                {"type": "delta", "mixer": delta, "mlp": moe}, {"type": "attention", "mixer": attn, "mlp": moe}]}


def time_parts(engine, s: dict, lens_before: list, new_tokens: int, peaks: dict, timer: Timer) -> dict:
    """Milliseconds of the Pagulix model's mixers and feed-forward and of their kernels alone, for a step of `new_tokens`
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
    i32 = lambda k: torch.zeros(k, dtype=torch.int32, device=dev)

    # ---- the streams: a sublayer's result written, the next one's input read and normed --------------------------------
    S, link, norm, scale = s["streams"], blocks[0].feed_forward_link, blocks[0].feed_forward_norm, blocks[0].mixer_scale
    streams = torch.randn(n, S * width, device=dev)
    branch, normed = torch.zeros(n, width, device=dev), torch.empty(n, width, dtype=bf, device=dev)
    border = dict(scale=scale.weight, mix=link.mix, write=link.write_scaled, read=link.read, norm=norm.factor, eps=norm.eps, out=normed)
    row("streams_write_read_norm", timer(lambda: ops.streams_step(streams, S, branch=branch, **border)), 0.0,
        n * width * (8 * S + 8 + 2) + width * 8)

    # ---- latent attention over a window (layer 0) ------------------------------------------------------------------------
    lat, cache0 = blocks[0].mixer, engine.cache.layer(0)
    H, d, rd, vd, rank, window = s["lheads"], s["ldim"], s["lrot"], s["lvdim"], s["rank"], s["window"]
    wide = rank + rd
    out["latent_mixer_ms"] = round(timer(lambda: lat.forward(x, residual, ctx, cache0, True)), 4)
    vis = rows_read = 0
    for before in lens_before:
        vis += sum(min(window, p + 1) for p in range(before, before + new_tokens))
        rows_read += before + new_tokens - max(0, before - window + 1)
    q_wide = (torch.randn(n, H * wide, device=dev) * 0.3).to(bf)
    o_lat = torch.empty(H * n, rank, dtype=bf, device=dev)
    ms = timer(lambda: attn_kernels.latent_attention(q_wide, cache0, o_lat, ctx, n_heads=H, key_dim=wide, rank=rank, scale=lat.scale,
                                                     window=window, sink=lat.sinks))
    row("latent_attention", ms, 2.0 * (wide + rank) * vis * H, rows_read * wide * 2 + n * H * (wide + rank) * 2)
    tile_rows = tcgen05.GROUPED_TILE_ROWS
    if not (tcgen05.grouped_supports(bf, lat.w_uk_t) and tcgen05.grouped_supports(bf, lat.w_uv)):
        raise RuntimeError("the benchmark's latent products run on the tensor cores")
    offsets, order, tiles, n_tiles = i32(H + 1), i32(H * n), i32(2 * H * (-(-n // tile_rows))), i32(1)
    proj = (torch.randn(n, lat.w_in.n, device=dev) * 0.3).to(bf)
    q_nope = torch.empty(H * n, d, dtype=bf, device=dev)
    pos = lat.position
    row("latent_prepare", timer(lambda: ops.latent_prepare(
        proj, pos.cos, pos.sin, lat.latent_norm, lat.eps, ctx.token_pos, ctx.token_seq, ctx.seq_slot, ctx.page_table, cache0.k, q_nope,
        q_wide, offsets, order, tiles, n_tiles, n_heads=H, head_dim=d, rot_dim=rd, rank=rank, rot_dims=pos.rot_dims, style=pos.style,
        page_size=ctx.page_size, write_kv=True, tile_rows=tile_rows)), 0.0, n * (H * (d + rd) * 2 + wide * 2) * 2)
    v = torch.empty(H * n, vd, dtype=f32, device=dev)
    row("queries_into_latent", timer(lambda: tcgen05.grouped_gemm_spread(q_nope, lat.w_uk_t, q_wide, wide, offsets, tiles, n_tiles, n_pairs=H * n)),
        2.0 * n * H * d * rank, H * d * rank * 2 + n * H * (d * 2 + rank * 2))
    row("latents_to_values", timer(lambda: lat._grouped(o_lat, lat.w_uv, v, (offsets, order, tiles, n_tiles, True), H * n)),
        2.0 * n * H * vd * rank, H * vd * rank * 2 + n * H * (rank * 2 + vd * 4))
    plain = torch.empty(n, H * vd, dtype=bf, device=dev)
    row("latent_gate", timer(lambda: ops.latent_gate(v, None, plain, n_tokens=n, n_heads=H, v_head_dim=vd)), 0.0, n * H * vd * 6)
    del q_wide, o_lat, proj, q_nope, v, plain

    # ---- attention with values of their own size, blended with the first such layer's (layer 3) ---------------------------------
    att, cache3 = blocks[3].mixer, engine.cache.layer(3)
    hd, vhd, heads, kv = s["hd"], s["vd"], s["heads"], s["kv"]
    ctx.extras["first_values"] = (torch.randn(n, att.w_qkv.n, device=dev).to(bf), att.q_dim + att.kv_dim, att.v_dim)
    first_rows = ctx.extras["first_values"][0]
    out["attention_mixer_ms"] = round(timer(lambda: att.forward(x, residual, ctx, cache3, True)), 4)
    causal = sum(p + 1 for before in lens_before for p in range(before, before + new_tokens))
    keys = sum(before + new_tokens for before in lens_before)
    qkv = torch.randn(n, att.w_qkv.n, device=dev).to(bf)
    mixed = torch.empty(n, att.o_dim, dtype=bf, device=dev)
    ms = timer(lambda: attn_kernels.attention(qkv, cache3, mixed, ctx, n_heads=heads, n_kv_heads=kv, head_dim=hd, scale=att.scale, v_head_dim=vhd))
    row("attention", ms, 2.0 * (hd + vhd) * causal * heads, keys * kv * (hd + vhd) * 2 + n * heads * (hd + vhd) * 2)
    ms = timer(lambda: att.position.apply_normed_and_store(
        qkv, ctx, cache3, n_heads=heads, n_kv_heads=kv, head_dim=hd, write_kv=True, q_weight=att.q_norm, k_weight=att.k_norm, eps=1e-5,
        v_head_dim=vhd, value_mix=(att.value_lambda, first_rows, att.q_dim + att.kv_dim)))
    row("norm_rotate_blend_store", ms, 0.0, n * (2 * heads * hd + 2 * kv * hd + 3 * kv * vhd) * 2)
    qkv_acc = torch.zeros(n, att.w_qkv.n, dtype=f32, device=dev)
    project = ((lambda: linear.accumulate_split(x, att.w_qkv, qkv_acc, ctx)) if linear.wants_split(x, att.w_qkv)      # as the part calls it
               else (lambda: linear.project(x, att.w_qkv, qkv, ctx)))
    row("qkv_projection", timer(project), 2.0 * n * att.w_qkv.n * width,
        att.w_qkv.n * width * 2 + n * (width + att.w_qkv.n) * 2)

    # ---- the delta rule (layer 2) ------------------------------------------------------------------------------------------------
    rule, cache2 = blocks[2].mixer, engine.cache.layer(2)
    out["delta_mixer_ms"] = round(timer(lambda: rule.forward(x, residual, ctx, cache2, True)), 4)
    matrix, conv = cache2.parts
    H, G, dim, vdim = rule.n_heads, rule.n_kv_heads, rule.head_dim, rule.v_head_dim
    z = torch.randn(n, rule.width, device=dev) * 0.5
    u = torch.empty(n, -(-(rule.conv_ch + 2 * H) // 4) * 4, dtype=f32, device=dev)
    ms = timer(lambda: ops.scan_prepare(
        z, conv_col=0, conv_ch=rule.conv_ch, taps=rule.w_conv, conv_bias=None, conv_state=conv.state, unit_heads=2 * G, unit_dim=dim,
        scaled_heads=G, unit_scale=dim ** -0.5, heads=H, decay_col=rule.a_col, step_col=rule.beta_col, a_log=rule.a_log,
        dt_bias=rule.dt_bias, out=u, cu_seqlens=ctx.cu_seqlens, token_seq=ctx.token_seq, seq_slot=ctx.seq_slot, n_seqs=ctx.n_seqs,
        longest_run=ctx.max_new))
    row("delta_prepare", ms, 0.0, n * (rule.conv_ch * 8 + 4 * H * 4) + 2 * B * conv.state[0].numel() * 4)
    o = torch.empty(n, rule.v_dim, dtype=f32, device=dev)
    ms = timer(lambda: ops.state_scan(u, matrix.state, o, ctx.cu_seqlens, ctx.seq_slot, n_seqs=ctx.n_seqs, heads=H, groups=G, dim=dim,
                                      vdim=vdim, q_col=0, k_col=rule.qk_dim, v_col=2 * rule.qk_dim, decay_col=rule.conv_ch,
                                      step_col=rule.conv_ch + H, delta=True, longest_run=ctx.max_new))
    row("delta_scan", ms, 0.0, n * (H * (2 * dim + vdim + 2) + H * vdim) * 4 + 2 * B * H * dim * vdim * 4, fp32_flops=8.0 * n * H * dim * vdim)
    gated = torch.empty(n, rule.v_dim, dtype=bf, device=dev)
    ms = timer(lambda: ops.gated_group_norm(o, z, rule.gate_col, rule.norm, gated, groups=H, group_size=vdim, gate_first=False, eps=1e-5))
    row("delta_gated_norm", ms, 0.0, n * H * vdim * (4 + 4 + 2))
    row("delta_projection", timer(lambda: linear.logits(x, rule.w_in, z, ctx)), 2.0 * n * rule.width * width,
        rule.width * width * 2 + n * (width * 2 + rule.width * 4))
    del z, u, o, gated

    # ---- experts -------------------------------------------------------------------------------------------------------------------
    mx = blocks[0].feed_forward
    out["experts_feed_forward_ms"] = round(timer(lambda: mx.forward(x, residual, ctx)), 4)
    # a step of few tokens lists the shared expert's slices as experts that every token uses; else they are matrices of their own
    extra = mx.in_lists if n <= mx.SHARED_IN_LISTS_TOKENS else 0
    chosen, top, experts, f, shared = mx.top, mx.top + extra, mx.n_experts + extra, mx.expert_size, mx.shared_size
    pairs = n * top
    ids, wts = torch.empty(n, top, dtype=torch.int32, device=dev), torch.empty(n, top, dtype=f32, device=dev)
    row("router", timer(lambda: ops.moe_route(x, mx.router, None, ids, wts, top=chosen, always=extra, softmax=True, bias=mx.router_bias,
                                              **mx.route_cut(x, ctx))),
        0.0, mx.n_experts * width * 4 + n * width * 2, fp32_flops=2.0 * n * mx.n_experts * width)
    used = int(torch.unique(ids).numel())
    if not mx._on_tensor_cores(x):
        raise RuntimeError("the benchmark's experts run on the tensor cores")
    offsets, order, tiles, n_tiles, place = i32(experts + 1), i32(pairs), i32(2 * (-(-pairs // tile_rows) + experts)), i32(1), i32(pairs)
    arrange = lambda: ops.moe_arrange(ids, pairs, experts, tile_rows, offsets, order, tiles, n_tiles, place)
    arrange()
    y = torch.randn(pairs, width, dtype=f32, device=dev)
    acts = torch.empty(pairs, f, dtype=bf, device=dev)
    xs = torch.zeros(pairs, width, dtype=bf, device=dev)
    gather = lambda: ops.moe_gather(x, xs, order, n_pairs=pairs, top=top)
    gather()
    w_gate, w_up, w_down = mx.w_gate[:experts], mx.w_up[:experts], mx.w_down[:experts]
    ms_up = timer(lambda: tcgen05.grouped_gemm(xs, w_gate, w_up, acts, offsets, tiles, n_tiles, n_pairs=pairs))
    ms_down = timer(lambda: tcgen05.grouped_gemm(acts, w_down, None, y, offsets, tiles, n_tiles, n_pairs=pairs))
    out["gather_ms"], out["arrange_ms"] = round(timer(gather), 4), round(timer(arrange), 4)
    row("experts_gate_up", ms_up, 2.0 * pairs * 2 * f * width, used * 2 * f * width * 2 + pairs * (width + f) * 2)
    row("experts_down", ms_down, 2.0 * pairs * f * width, used * f * width * 2 + pairs * (f * 2 + width * 4))
    shared_y = None
    if not extra:
        w_gate, w_up, w_down = mx.shared
        sact, shared_y = torch.empty(n, shared, dtype=bf, device=dev), torch.empty(n, width, dtype=f32, device=dev)
        row("shared_gate_up", timer(lambda: linear.gated(x, w_gate, w_up, sact, ctx)), 2.0 * n * 2 * shared * width,
            2 * shared * width * 2 + n * (width + shared) * 2)
        row("shared_down", timer(lambda: linear.logits(sact, w_down, shared_y, ctx)), 2.0 * n * shared * width,
            shared * width * 2 + n * (shared * 2 + width * 4))
    left = dict(y=y, weights=wts, top=top, place=place, shared=shared_y, factor=1.0)
    row("experts_sum_streams_write_read_norm", timer(lambda: ops.streams_step(streams, S, experts=left, **border)), 0.0,
        pairs * (width * 4 + 8) + n * width * (8 * S + 2 + (0 if extra else 4)) + width * 8)
    out["experts_used"] = used
    engine.workspace.rezero()
    for slot in slots:
        engine.free_slot(slot)
    return out


def dense_qkv(engine, s: dict, lens_before: list, new_tokens: int, peaks: dict, timer: Timer) -> dict:
    """The dense decoder's q, k, v projection alone, as its mixer calls it."""
    from . import linear
    slots, ctx = _step_context(engine, lens_before, new_tokens, s["vocab"], 5)
    n, w, dev = ctx.n_tokens, engine.model.layers[0].block.mixer.w_qkv, engine.device
    x = (torch.randn(n, w.k, device=dev) * 0.5).to(torch.bfloat16)
    split = linear.wants_split(x, w)
    out = torch.zeros(n, w.n, dtype=torch.float32 if split else torch.bfloat16, device=dev)
    ms = timer((lambda: linear.accumulate_split(x, w, out, ctx)) if split else (lambda: linear.project(x, w, out, ctx)))
    ideal = _roofline_ms(2.0 * n * w.n * w.k, w.n * w.k * 2 + n * (w.k * 2 + w.n * out.element_size()), peaks)
    for slot in slots:
        engine.free_slot(slot)
    return {"qkv_projection": {"ms": round(ms, 4), "roofline_ms": round(ideal, 6), "x_roofline": round(ms / ideal, 2)}}


# how far each kernel of the design is from its roofline, over the like kernel of the closest model
LIKE = {"streams_write_read_norm": ("dense", "rms_norm"), "experts_sum_streams_write_read_norm": ("dense", "rms_norm"), "latent_attention": ("vadodra", "latent_attention"),
        "latent_prepare": ("vadodra", "latent_prepare"), "queries_into_latent": ("vadodra", "queries_into_latent"),
        "latents_to_values": ("vadodra", "latents_to_values"), "latent_gate": ("vadodra", "latent_gate"),
        "attention": ("dense", "attention"), "norm_rotate_blend_store": ("vadodra", "norm_rotate_store"),
        "qkv_projection": ("dense", "qkv_projection"), "delta_projection": ("dense", "down"),
        "delta_prepare": ("redodra", "delta_rule_prepare"), "delta_scan": ("redodra", "delta_rule_scan"),
        "delta_gated_norm": ("redodra", "delta_rule_gated_norm"), "experts_gate_up": ("lulisun", "experts_gate_up"),
        "experts_down": ("lulisun", "experts_down"), "shared_gate_up": ("dense", "gate_up"), "shared_down": ("dense", "down")}


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
    result = {"arch": "pagulix", "sizes": sizes, "config": s, "dtype": "bf16", "data": "synthetic (random weights, random token ids)",
              "peaks": dict(peaks, source=peak_source), "l2": "256 MiB written between timed iterations"}
    ls, vs = redodra_bench._lulisun_sizes(s), vadodra_bench.SIZES[sizes]
    models = (("pagulix", pagulix_config(s)), ("vadodra", vadodra_bench.vadodra_config(vs)), ("redodra", redodra_bench.redodra_config(s)),
              ("lulisun", arch_bench.lulisun_config(ls)), ("dense", redodra_bench.dense_config(s, cache_tokens)))
    for kind, cfg in models:
        t0 = time.time()
        engine = Engine.from_random(config_from_dict(cfg), seed=0, std=0.02, dtype="bfloat16", device="cuda:0",
                                    max_tokens=cache_tokens, n_slots=batch + 2)
        print(f"[bench] {kind} ready in {time.time() - t0:.1f} s", file=sys.stderr, flush=True)
        r = throughput(engine, s, prefill_tokens=prefill_tokens, batch=batch, context=context, steps=steps, timer=timer)
        for phase, before, new in (("prefill_parts", [0], prefill_tokens), ("decode_parts", [context] * batch, 1)):
            if kind == "pagulix":
                r[phase] = time_parts(engine, s, before, new, peaks, timer)
            elif kind == "vadodra":
                r[phase] = vadodra_bench.time_parts(engine, vs, before, new, peaks, timer)
            elif kind == "redodra":
                r[phase] = redodra_bench.time_parts(engine, s, before, new, peaks, timer)
            elif kind == "lulisun":
                r[phase] = arch_bench.time_parts(engine, "lulisun", ls, before, new, peaks, timer)
            else:
                r[phase] = arch_bench.time_parts(engine, "dense", s, before, new, peaks, timer)
                r[phase].update(dense_norm_and_rope(engine, s, before, new, peaks, timer))
                r[phase].update(dense_qkv(engine, s, before, new, peaks, timer))
        engine.check_device_status()
        result[kind] = r
        del engine
        torch.cuda.empty_cache()
    ratios = {}
    for phase in ("prefill_parts", "decode_parts"):
        for name, (model, other) in LIKE.items():
            if name in result["pagulix"][phase]:
                ratios[f"{phase[:-6]}.{name} (over {model} {other})"] = round(
                    result["pagulix"][phase][name]["x_roofline"] / result[model][phase][other]["x_roofline"], 2)
        for name, other in (("router", "route_ms"),):
            ratios[f"{phase[:-6]}.{name} ms (over lulisun {name} ms)"] = round(
                result["pagulix"][phase][name]["ms"] / max(result["lulisun"][phase][other], 1e-6), 2)
    result["x_roofline_over_like"] = ratios
    print(json.dumps(result))
    return 0
