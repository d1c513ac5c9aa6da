"""Prefill and decode throughput of the Dizepel design at layer sizes that resemble a real model's, beside the Fivedra design's
parallel layers (attention beside a matrix memory: the engine's closest other model) and the Llama shape at equal width, layer
count and parameters, and the design's kernels alone beside the like kernel of those models.

    python bench.py --design dizepel [--steps K] [--warmup W]

Random weights, seeded random token ids.  Timing as in bench.py: CUDA events on the launching stream after warm-up;
decode steps read weights and caches far larger than L2; prefill and the kernels alone start from a flushed L2.
"""
from __future__ import annotations

import json

import torch

from .design_bench import BLOCK_SIZE, CONTEXT, PREFILL_TOKENS, llama_config, measure_model
from .fivedra_bench import fivedra_config


def dizepel_config(width, heads, kv_heads, dim, ssm_heads, vdim, state, groups, ff, vocab, layers=4):
    pair = {"type": "parallel", "mlp": {"kind": "dense", "ff": ff},
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5 / 8, "conv": 4, "softcap": 30.0,
                               "rot": {"dims": dim // 2, "base": 5.0e5, "scaling": {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}}},
                      "right": {"heads": ssm_heads, "vdim": vdim, "state": state, "groups": groups, "conv": 4, "norm_groups": groups}}}
    return {"architecture": "Dizepel", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5}, "canon": {"taps": 4},
            "loop": {"start": 0, "stop": layers, "times": 1}, "layers": [pair] * layers}


def parallel_only(cfg):
    return dict(cfg, layers=[cfg["layers"][0]] * 4)


# name -> (Dizepel, Fivedra with parallel layers only, Llama), of one width, layer count and about the same parameters
SIZES = {
    "width2048": (dizepel_config(2048, 16, 4, 128, 32, 64, 128, 4, 4096, 32000),
                  parallel_only(fivedra_config(2048, 16, 4, 128, 1024, 4, 128, 256, 768, 5632, 32000)),
                  llama_config(2048, 16, 4, 128, 4864, 32000, 4)),
    "width4096": (dizepel_config(4096, 32, 8, 128, 64, 64, 128, 8, 8192, 32000),
                  parallel_only(fivedra_config(4096, 32, 8, 128, 1024, 8, 128, 256, 1536, 11264, 32000)),
                  llama_config(4096, 32, 8, 128, 9984, 32000, 4)),
}


def kernels_alone(pk, width=4096, heads=32, kv_heads=8, dim=128, sh=64, sdv=64, state=128, groups=8, ff=8192, taps=4):
    """Each new kernel, or kernel that gained a branch, alone with the like kernel beside it, and what each reaches of its
    roofline: the measured copy rate for kernels that stream, the measured bf16 product rate for the tensor-core attention kernels
    (the products that the mask leaves), the nominal float32 FMA rate (148 SMs x 128 lanes x 2 x 1.9 GHz) over the operations of
    the recurrence (5 per token and cell of the state) for the float32 scans of a prompt."""
    from lmsf_b200 import kernels
    from lmsf_b200.benchmarks.kernel_bench import Timer
    dev = torch.device("cuda:0")
    tm = Timer(dev)
    bf, f32, i32 = torch.bfloat16, torch.float32, torch.int32
    T, B = PREFILL_TOKENS, 64
    hbm, tflops, fp32 = pk["hbm_gbs"] * 1e9, pk["bf16_tflops"] * 1e12, 148 * 128 * 2 * 1.9e9
    rows = {}

    def rec(name, sec, bytes_=None, flops=None, fma=None, like=None):
        r = {"us": round(sec * 1e6, 1)}
        if bytes_ is not None:
            r["frac_of_copy_rate"] = round(bytes_ / sec / hbm, 3)
        if flops is not None:
            r["frac_of_bf16_peak"] = round(flops / sec / tflops, 4)
        if fma is not None:
            r["frac_of_fp32_peak"] = round(fma / sec / fp32, 4)
        if like:
            r["like"] = like
        rows[name] = r

    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s, dtype=bf, scale=1.0: (torch.randn(*s, generator=g, device=dev, dtype=f32) * scale).to(dtype)
    ones = lambda n: torch.ones(n, device=dev)
    ints = lambda v: torch.tensor(v, dtype=i32, device=dev)
    H, G, bs = heads, kv_heads, BLOCK_SIZE
    pos, cu, ctxl, slot, flag = torch.arange(T, dtype=i32, device=dev), ints([0, T]), ints([T]), ints([0]), ints([0])
    seq = ints([0] * T)
    cud, ctxd, slotd = torch.arange(B + 1, dtype=i32, device=dev), ints([CONTEXT] * B), torch.arange(B, dtype=i32, device=dev)
    # ---- what lies between two branches
    res, y1, y2, h, w = rnd(T, width, dtype=f32), rnd(T, width), rnd(T, width), torch.empty(T, width, dtype=bf, device=dev), ones(width)
    norms = dict(w_post=w, eps_post=1e-5, post_centred=True, h=h, w_next=w, eps_next=1e-5, next_centred=True)
    rec(f"stream_layer (pair joined, layer norm, add, next layer norm) 2048 x {width}",
        tm.run(lambda: kernels.stream_layer(res, y=y1, pair=(y2, w, w, 1e-5, 0.5), **norms), 3, 10), bytes_=T * width * 14, like="stream_norm below")
    rec(f"stream_layer (layer norm, add, next layer norm) 2048 x {width}", tm.run(lambda: kernels.stream_layer(res, y=y1, **norms), 3, 10),
        bytes_=T * width * 12, like="stream_norm below")
    rec(f"stream_norm (Vufolorn: post norm, layer scale, add, next norm) 2048 x {width}",
        tm.run(lambda: kernels.stream_norm(res, y=y1, w_post=w, layer_scale=w, eps_post=1e-5, h=h, w_next=w, eps_next=1e-5), 3, 10), bytes_=T * width * 12)
    filt, fst = rnd(width, taps, dtype=f32), torch.zeros(B + 1, (taps - 1) * width, device=dev)
    r64, a64, b64, h64 = rnd(B, width, dtype=f32), rnd(B, width), rnd(B, width), torch.empty(B, width, dtype=bf, device=dev)
    n64 = dict(norms, h=h64)
    rec(f"stream_layer (pair, norms, filter of {taps} taps) 64 single tokens x {width}",
        tm.run(lambda: kernels.stream_layer(r64, y=a64, pair=(b64, w, w, 1e-5, 0.5), filt=(filt.t().contiguous(), fst, slotd), **n64), 3, 10),
        bytes_=B * width * (14 + 8 * (taps - 1)), like="stream_norm of 64 rows below")
    rec(f"stream_norm (Vufolorn) 64 single tokens x {width}",
        tm.run(lambda: kernels.stream_norm(r64, y=a64, w_post=w, layer_scale=w, eps_post=1e-5, h=h64, w_next=w, eps_next=1e-5), 3, 10), bytes_=B * width * 12)
    rec(f"causal_conv with the input added ({taps} taps) 2048 x {width}",
        tm.run(lambda: kernels.causal_conv(h, y1, filt, None, fst, 0, cu, slot, 1, T, act="add_input"), 3, 10), bytes_=T * width * 4, like="token_shift below")
    st1 = torch.zeros(B + 1, width, device=dev)
    rec(f"token_shift (Zonidra) 2048 x {width}", tm.run(lambda: kernels.token_shift(h, y1, w, st1, pos, seq, cu, slot), 3, 10), bytes_=T * width * 4)
    z, zo, coef = rnd(T, ff), torch.empty(T, ff, dtype=bf, device=dev), rnd(4, dtype=f32)
    rec(f"poly_norm 2048 x {ff}", tm.run(lambda: kernels.poly_norm(zo, z, coef, 1e-5), 3, 10), bytes_=T * ff * 4, like="gated_act below")
    gu = rnd(T, 2 * ff)
    rec(f"gated_act (Llama, silu) 2048 x {ff}", tm.run(lambda: kernels.gated_act(zo, gu, "silu"), 3, 10), bytes_=T * ff * 6)
    # ---- queries and keys on their way into attention
    pages = T // bs
    C = (H + G) * dim
    tab = torch.arange(pages, dtype=i32, device=dev).view(1, pages)
    c2 = rnd(pages + 1, 2, G, bs, dim, scale=0.5)
    x, q = rnd(T, C), torch.empty(T, H * dim, dtype=bf, device=dev)
    wt, cst = rnd(taps, C, dtype=f32), torch.zeros(B + 1, (taps - 1) * C, device=dev)
    inv = torch.tensor([1.0e4 ** (-4.0 * i / dim) for i in range(dim // 4)], dtype=f32, device=dev)
    rec(f"conv_rope_cache_write ({taps} taps, {dim // 2} of {dim} values turned) 2048 tokens, {H} + {G} heads",
        tm.run(lambda: kernels.conv_rope_cache_write(q, x, wt, cst, 0, cu, slot, pos, tab, bs, c2, inv, dim // 2, 1.2, H, G, dim, 1, T, flag), 3, 10),
        bytes_=T * (2 * C + G * dim) * 2, like="rope_cache_write below")
    kc, vc = rnd(T, G * dim), rnd(T, G * dim)
    inv_l = torch.tensor([1.0e4 ** (-2.0 * i / dim) for i in range(dim // 2)], dtype=f32, device=dev)
    rec(f"rope_cache_write (Llama) 2048 tokens, {H} + {G} heads",
        tm.run(lambda: kernels.rope_cache_write(q, kc, vc, pos, seq, tab, bs, c2, inv_l, dim, True, H, G, dim, flag), 3, 10), bytes_=T * (2 * C + 2 * G * dim) * 2)
    pages_d = B * (CONTEXT // bs)
    tabd = torch.arange(pages_d, dtype=i32, device=dev).view(B, CONTEXT // bs)
    posd, seqd = ints([CONTEXT - 1] * B), torch.arange(B, dtype=i32, device=dev)
    cd = rnd(pages_d, 2, G, bs, dim, scale=0.5)
    xd, qd = rnd(B, C), torch.empty(B, H * dim, dtype=bf, device=dev)
    rec(f"conv_rope_cache_write, 64 single tokens, {H} + {G} heads",
        tm.run(lambda: kernels.conv_rope_cache_write(qd, xd, wt, cst, 0, cud, slotd, posd, tabd, bs, cd, inv, dim // 2, 1.2, H, G, dim, B, 1, flag), 3, 10),
        bytes_=B * ((2 * C + G * dim) * 2 + (taps - 1) * C * 8), like="rope_cache_write of 64 below")
    rec(f"rope_cache_write (Llama), 64 single tokens, {H} + {G} heads",
        tm.run(lambda: kernels.rope_cache_write(qd, kc[:B], vc[:B], posd, seqd, tabd, bs, cd, inv_l, dim, True, H, G, dim, flag), 3, 10),
        bytes_=B * (2 * C + 2 * G * dim) * 2)
    # ---- attention with capped scores and a sink
    t128 = torch.arange(0, T, 128, dtype=i32, device=dev).flip(0).contiguous()
    t64 = torch.arange(0, T, 64, dtype=i32, device=dev).flip(0).contiguous()
    s128, s64 = torch.zeros_like(t128), torch.zeros_like(t64)
    flops, scale = 4.0 * (T * (T + 1) // 2) * dim * H, dim ** -0.5
    qf, o, sink = rnd(T, H * dim), torch.empty(T, H * dim, dtype=bf, device=dev), torch.zeros(H, device=dev)
    tc = lambda qq, **ex: tm.run(lambda: kernels.attention_prefill_tc(o, qq, c2, tab, bs, s128, t128, t128.numel(), cu, ctxl, scale, 0, H, G, dim, flag, **ex), 3, 10)
    mma = lambda qq, **ex: tm.run(lambda: kernels.attention_prefill(o, qq, c2, tab, bs, s64, t64, t64.numel(), cu, ctxl, scale, 0, H, G, dim, **ex), 3, 10)
    own, name = dict(sinks=sink, softcap=30.0), f"2048 tokens, {H} heads of {dim} over {G}"
    rec(f"attention_prefill_tc, capped scores, sink: {name}", tc(qf, **own), flops=flops, like="the plain one below")
    rec(f"attention_prefill_tc, capped scores far from zero (no series), sink: {name}", tc(qf * 40, **own), flops=flops, like="the plain one below")
    rec(f"attention_prefill_tc (Llama) {name}", tc(qf), flops=flops)
    rec(f"attention_prefill (mma.sync), capped scores, sink: {name}", mma(qf, **own), flops=flops, like="the plain one below")
    rec(f"attention_prefill (mma.sync, plain) {name}", mma(qf), flops=flops)
    splits, warps = kernels.decode_plan(B, G, H // G, CONTEXT, dim, kernels.decode_widths(dim, H // G))
    need = kernels.attention_decode_scratch_floats(B, H, splits, dim)
    scratch, od = torch.zeros(max(need, 1), dtype=f32, device=dev), torch.empty(B, H * dim, dtype=bf, device=dev)
    qd = rnd(B, H * dim)
    for what, ex in (("capped scores, sink", own), ("Llama", {})):
        rec(f"attention_decode ({what}) 64 requests at 2048, {H} heads of {dim} over {G}",
            tm.run(lambda: kernels.attention_decode(od, qd, cd, tabd, bs, None, B, cud, ctxd, scale, 0, H, G, dim, splits, scratch if need else None, warps, **ex), 3, 10),
            bytes_=B * CONTEXT * G * dim * 4, like="the plain one below" if ex else None)
    # ---- the state space
    inner, ch = sh * sdv, sh * sdv + 2 * groups * state
    xb, cb = rnd(T, ch), torch.empty(T, ch, dtype=bf, device=dev)
    cw, cbias, cs2 = rnd(ch, taps, dtype=f32), ones(ch), torch.zeros(B + 1, (taps - 1) * ch, device=dev)
    rec(f"causal_conv (silu) 2048 x {ch}", tm.run(lambda: kernels.causal_conv(cb, xb, cw, cbias, cs2, 0, cu, slot, 1, T, act="silu"), 3, 10),
        bytes_=T * ch * 4, like="token_shift above")
    dtr, yo = rnd(T, sh), torch.empty(T, inner, dtype=f32, device=dev)
    a_log, dtb, skip = torch.zeros(sh, device=dev), torch.full((sh,), -3.0, device=dev), ones(sh)
    cells = sh * sdv * state
    sst = torch.zeros(B + 1, cells, device=dev)
    kk, qq, vv = xb[:, inner:inner + groups * state], xb[:, inner + groups * state:], xb[:, :inner]
    n_c = kernels.scan_chunk_tokens()
    chunks = [(0, c, min(c + n_c, T), j) for j, c in enumerate(range(0, T, n_c))]
    items, spans = ints(chunks), ints([(0, 0, len(chunks), 0)])
    ends = (dtb, a_log, skip, sst)
    rec(f"scan_chunks (three launches), a prompt of 2048 tokens, {sh} heads of {state} x {sdv}",
        tm.run(lambda: kernels.scan_chunks(yo, qq, kk, vv, dtr, *ends, cu, slot, 1, sh, groups, state, sdv, items=items, spans=spans), 3, 10),
        fma=5.0 * T * cells, like="gated_scan and matrix_memory below")
    rec(f"gated_scan (Redarax: one chain of tokens), a prompt of 2048 tokens, {sh} heads of {state} x {sdv}",
        tm.run(lambda: kernels.gated_scan(yo, qq, kk, vv, dtr, None, *ends, cu, slot, 1, sh, groups, state, sdv, delta=False, k_times_dt=True), 3, 10),
        fma=5.0 * T * cells)
    mh, mdk, mdv = 8, 128, 256
    QK, V = mh * mdk, mh * mdv
    p = rnd(T, 2 * QK + V + 2 * mh)
    mst, mo = torch.zeros(B + 1, kernels.matrix_memory_state_floats(mh, mdk, mdv), device=dev), torch.empty(T, V, dtype=f32, device=dev)
    zero, last = torch.zeros(mh, device=dev), ints([0] * (len(chunks) - 1) + [1])
    rec(f"matrix_memory (Fivedra, three launches), a prompt of 2048 tokens, {mh} heads of {mdk} x {mdv}",
        tm.run(lambda: kernels.matrix_memory(mo, p[:, :QK], p[:, QK:2 * QK], p[:, 2 * QK:2 * QK + V], p[:, 2 * QK + V:2 * QK + V + mh], p[:, 2 * QK + V + mh:],
                                             zero, zero, mst, cu, slot, 1, mh, mdk, mdv, 15.0, mdk ** -0.5, items=items, spans=spans, last_chunk=last), 3, 10),
        fma=5.0 * T * mh * mdk * mdv)
    y64 = torch.empty(B, inner, dtype=f32, device=dev)
    step = (qq[:B], kk[:B], vv[:B], dtr[:B])
    rec(f"scan_chunks of single tokens (one launch), 64 requests, {sh} heads of {state} x {sdv}",
        tm.run(lambda: kernels.scan_chunks(y64, *step, *ends, cud, slotd, B, sh, groups, state, sdv), 3, 10), bytes_=B * cells * 8, like="the two below")
    rec(f"gated_scan (Redarax, two launches) 64 single tokens, {sh} heads of {state} x {sdv}",
        tm.run(lambda: kernels.gated_scan(y64, *step, None, *ends, cud, slotd, B, sh, groups, state, sdv, delta=False, k_times_dt=True), 3, 10),
        bytes_=B * cells * 8)
    rec(f"matrix_memory (Fivedra) 64 single tokens, {mh} heads of {mdk} x {mdv}",
        tm.run(lambda: kernels.matrix_memory(mo[:B], p[:B, :QK], p[:B, QK:2 * QK], p[:B, 2 * QK:2 * QK + V], p[:B, 2 * QK + V:2 * QK + V + mh],
                                             p[:B, 2 * QK + V + mh:], zero, zero, mst, cud, slotd, B, mh, mdk, mdv, 15.0, mdk ** -0.5), 3, 10),
        bytes_=B * mh * mdk * mdv * 8)
    gate, yn = rnd(T, inner), torch.empty(T, inner, dtype=bf, device=dev)
    rec(f"grouped_gated_norm (gate first, {groups} parts) 2048 x {inner}",
        tm.run(lambda: kernels.grouped_gated_norm(yn, yo, gate, ones(inner), inner // groups, 1e-5, gate_act="silu", gate_first=True), 3, 10),
        bytes_=T * inner * 8, like="gated_norm below")
    rec(f"gated_norm (Vufolorn: one norm a row) 2048 x {inner}", tm.run(lambda: kernels.gated_norm(yn, yo, gate, ones(inner), 1e-5), 3, 10), bytes_=T * inner * 8)
    return rows


def run(bench, steps, warmup, pk):
    sampler = bench.ClockSampler()
    sampler.start()
    sizes = {name: {m: measure_model(cfg, [8, 64], steps, warmup, bench) for m, cfg in zip(("dizepel", "fivedra_parallel", "llama"), cfgs)}
             for name, cfgs in SIZES.items()}
    alone = kernels_alone(pk)
    line = {"metric": "prefill and decode tokens/s of the Dizepel design beside the Fivedra design's parallel layers and the Llama shape of equal "
                      "width and parameters (4 layers each, random weights)",
            "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "dtype": "bf16", "data": "synthetic",
            "config": {"prefill_tokens": PREFILL_TOKENS, "context": CONTEXT, "block_size": BLOCK_SIZE,
                       "sizes": {k: v[0] for k, v in SIZES.items()}, "fivedra": {k: v[1] for k, v in SIZES.items()},
                       "llama": {k: v[2] for k, v in SIZES.items()}, "peaks": pk.get("source", "measured")},
            "sizes": sizes, "kernels_alone": alone, "clocks": sampler.stop(), "impl": "ours"}
    print(json.dumps(line))
    return 0
