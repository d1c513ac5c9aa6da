"""Prefill and decode throughput of the Fivedra design at layer sizes that resemble a real model's, beside the Vufolorn design
(the engine's other model of a recurrent mixer with a state matrix per head and attention over a cached low-rank vector) and
the Llama shape at equal width, layer count and about equal parameters per layer, and the design's kernels alone beside the
like kernel of those models.

    python bench.py --design fivedra [--steps K] [--warmup W]

Random weights, seeded random token ids.  Timing as in bench.py: CUDA events on the launching stream after warm-up;
decode steps read weights and caches far larger than L2; prefill and the kernels alone start from a flushed L2.
"""
from __future__ import annotations

import json

import torch

from . import design_bench
from .design_bench import BLOCK_SIZE, CONTEXT, PREFILL_TOKENS, measure_model


def fivedra_config(width, heads, kv_heads, dim, window, mem_heads, mem_dim, mem_vdim, q_rank, ff, vocab):
    mlp = {"kind": "dense", "ff": ff}
    pair = {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "bias_max": 256,
                               "mask": {"size": window}},
                      "right": {"heads": mem_heads, "dim": mem_dim, "vdim": mem_vdim, "gate_cap": 15.0},
                      "left_scale": 0.5, "right_scale": 0.75}}
    gru = {"type": "mingru", "mlp": mlp, "mixer": {"width": width}}
    lat = {"type": "latent_attention", "mlp": mlp,
           "mixer": {"heads": heads, "dim": dim, "rot_dim": 64, "vdim": dim, "kv_rank": 192, "q_rank": q_rank, "scale": (dim + 64) ** -0.5,
                     "rot": {"dims": 64, "base": 1.0e4, "scaling": {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}}
    return {"architecture": "Fivedra", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": width ** 0.5},
            "layers": [pair, gru, lat, pair]}


SIZES = {
    "width2048": fivedra_config(2048, 16, 4, 128, 1024, 4, 128, 256, 768, 4352, 32000),
    "width4096": fivedra_config(4096, 32, 8, 128, 1024, 8, 128, 256, 1536, 8192, 32000),
}


def kernels_alone(pk, width=4096, heads=32, kv_heads=8, dim=128, window=1024, mh=8, mdk=128, mdv=256, ff=8192):
    """Each new kernel, or kernel that gained a branch, alone with the like kernel beside it, and what each reaches of its
    roofline: the measured copy rate for kernels that stream, the measured bf16 product rate for the tensor-core attention
    kernels (the products that the mask leaves), the nominal float32 FMA rate (148 SMs x 128 lanes x 2 x 1.9 GHz) over the
    operations of the recurrence (5 per token and cell of the state) for the float32 scans of a prompt."""
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
    pos, seq, cu, ctxl, slot, flag = torch.arange(T, dtype=i32, device=dev), ints([0] * T), ints([0, T]), ints([T]), ints([0]), ints([0])
    cud, ctxd, slotd = torch.arange(B + 1, dtype=i32, device=dev), ints([CONTEXT] * B), torch.arange(B, dtype=i32, device=dev)
    # ---- the embedding, what ends a layer, the feed-forward's activation
    table, ids = rnd(32000, width), torch.randint(0, 32000, (T,), device=dev, generator=g).to(i32)
    res, xb = torch.empty(T, width, dtype=f32, device=dev), torch.empty(T, width, dtype=bf, device=dev)
    rec("embedding_stream (scaled row into the float32 stream) 2048 x 4096", tm.run(lambda: kernels.embedding_stream(res, table, ids, 64.0, flag), 3, 10),
        bytes_=T * width * 6, like="embedding below")
    rec("embedding (Llama) 2048 x 4096", tm.run(lambda: kernels.embedding(xb, table, ids, flag), 3, 10), bytes_=T * width * 4)
    y1, y2, h1, h2, w = rnd(T, width), rnd(T, width), torch.empty_like(xb), torch.empty_like(xb), ones(width)
    rec("stream_branches (two branches added, two norms) 2048 x 4096",
        tm.run(lambda: kernels.stream_branches(res, y1, 0.5, y2, 1.0, h1, w, h2, w, 1e-5), 3, 10), bytes_=T * width * 16, like="stream_norm below")
    rec("stream_norm (Vufolorn: post norm, layer scale, add, next norm) 2048 x 4096",
        tm.run(lambda: kernels.stream_norm(res, y=y1, w_post=w, layer_scale=w, eps_post=1e-5, h=h1, w_next=w, eps_next=1e-5), 3, 10), bytes_=T * width * 12)
    z, gu = rnd(T, ff), rnd(T, 2 * ff)
    rec(f"relu2_ (square of relu, in place) 2048 x {ff}", tm.run(lambda: kernels.relu2_(z), 3, 10), bytes_=T * ff * 4, like="gated_act below")
    rec(f"gated_act (Llama, silu) 2048 x {ff}", tm.run(lambda: kernels.gated_act(z, gu, "silu"), 3, 10), bytes_=T * ff * 6)
    # ---- the element-wise recurrence: three inputs and one output per token and channel
    p3, st = rnd(T, 3 * width), torch.zeros(B + 1, width, device=dev)
    rec("min_gru, a prompt of 2048 tokens x 4096",
        tm.run(lambda: kernels.min_gru(xb, p3[:, :width], p3[:, width:2 * width], p3[:, 2 * width:], w, w, st, cu, slot, 1, T), 3, 10),
        bytes_=T * width * 8, like="the prompt's scans below; gated_act above (three streams, one exponential)")
    pd, od_ = rnd(B, 3 * width), torch.empty(B, width, dtype=bf, device=dev)
    rec("min_gru, 64 single tokens x 4096",
        tm.run(lambda: kernels.min_gru(od_, pd[:, :width], pd[:, width:2 * width], pd[:, 2 * width:], w, w, st, cud, slotd, B, 1), 3, 10),
        bytes_=B * width * 16, like="matrix_memory and lightning_scan of single tokens below")
    # ---- the matrix memory against linear attention of the same state
    QK, V = mh * mdk, mh * mdv
    p = rnd(T, 2 * QK + V + 2 * mh)
    q, k, v, gi, gf = p[:, :QK], p[:, QK:2 * QK], p[:, 2 * QK:2 * QK + V], p[:, 2 * QK + V:2 * QK + V + mh], p[:, 2 * QK + V + mh:]
    bi, bf_ = torch.zeros(mh, device=dev), torch.full((mh,), 3.0, device=dev)
    mst = torch.zeros(B + 1, kernels.matrix_memory_state_floats(mh, mdk, mdv), device=dev)
    o = torch.empty(T, V, dtype=f32, device=dev)
    C = kernels.matrix_memory_chunk_tokens()
    chunks = [(0, c, min(c + C, T), j) for j, c in enumerate(range(0, T, C))]
    items, spans, last = ints(chunks), ints([(0, 0, len(chunks), 0)]), ints([0] * (len(chunks) - 1) + [1])
    cells = mh * mdk * mdv
    rec(f"matrix_memory (three launches), a prompt of 2048 tokens, {mh} heads of {mdk} x {mdv}",
        tm.run(lambda: kernels.matrix_memory(o, q, k, v, gi, gf, bi, bf_, mst, cu, slot, 1, mh, mdk, mdv, 15.0, mdk ** -0.5, items=items,
                                             spans=spans, last_chunk=last), 3, 10), fma=5.0 * T * cells, like="lightning below")
    lst, dec = torch.zeros(B + 1, mh, mdk, mdv, device=dev), torch.full((mh,), 0.98, device=dev)
    scr = torch.empty(len(chunks), mh, mdk, mdv, device=dev)
    la = (o, q, k, v, lst, dec, cu, slot, 1, mh, mdk, mdv, None)

    def lightning():
        kernels.lightning_scan(*la, items=items, scratch=scr, mode=1)
        kernels.lightning_prefix(scr, lst, dec, slot, items, spans)
        kernels.lightning_scan(*la, items=items, scratch=scr, mode=2)

    rec(f"lightning scan (Vufolorn, three launches), a prompt of 2048 tokens, {mh} heads of {mdk} x {mdv}", tm.run(lightning, 3, 10), fma=5.0 * T * cells)
    pd = rnd(B, 2 * QK + V + 2 * mh)
    qd, kd, vd, gid, gfd = pd[:, :QK], pd[:, QK:2 * QK], pd[:, 2 * QK:2 * QK + V], pd[:, 2 * QK + V:2 * QK + V + mh], pd[:, 2 * QK + V + mh:]
    o64 = torch.empty(B, V, dtype=f32, device=dev)
    rec(f"matrix_memory, 64 single tokens, {mh} heads of {mdk} x {mdv}",
        tm.run(lambda: kernels.matrix_memory(o64, qd, kd, vd, gid, gfd, bi, bf_, mst, cud, slotd, B, mh, mdk, mdv, 15.0, mdk ** -0.5), 3, 10),
        bytes_=B * cells * 8, like="lightning below")
    rec(f"lightning scan (Vufolorn), 64 single tokens, {mh} heads of {mdk} x {mdv}",
        tm.run(lambda: kernels.lightning_scan(o64, qd, kd, vd, lst, dec, cud, slotd, B, mh, mdk, mdv, None), 3, 10), bytes_=B * cells * 8)
    gate, yn = rnd(T, V), torch.empty(T, V, dtype=bf, device=dev)
    rec(f"grouped_gated_norm (norm per head of {mdv}, sigmoid gate, factor) 2048 x {V}",
        tm.run(lambda: kernels.grouped_gated_norm(yn, o, gate, ones(V), mdv, 1e-5, gate_act="sigmoid", out_scale=1.5), 3, 10), bytes_=T * V * 8,
        like="gated_norm below")
    rec(f"gated_norm (Vufolorn: one norm a row) 2048 x {V}", tm.run(lambda: kernels.gated_norm(yn, o, gate, ones(V), 1e-5), 3, 10), bytes_=T * V * 8)
    kernels_attention(rec, tm, rnd, ints, pos, seq, cu, ctxl, cud, ctxd, flag, T, B, H, G, dim, window)
    # ---- the products of a decode step
    x8 = rnd(8, width)
    extra = (2 * QK + 2 * V + 2 * mh + 15) // 16 * 16
    Wm, bias = rnd((H + G) * dim + extra, width, scale=0.02), rnd((H + G) * dim + extra)
    pages = 64
    c1, c2 = torch.zeros(pages, 1, G, bs, dim, dtype=bf, device=dev), torch.zeros(pages, 2, G, bs, dim, dtype=bf, device=dev)
    tab = torch.arange(8, dtype=i32, device=dev).view(8, 1)
    pos8, seq8 = ints([3] * 8), torch.arange(8, dtype=i32, device=dev)
    pm, qo = torch.empty(8, Wm.shape[0], dtype=bf, device=dev), torch.empty(8, H * dim, dtype=bf, device=dev)
    rec(f"gemm_skinny_qkv_rope, q and k with a bias, {extra} rows that pass: 8 x {Wm.shape[0]} x 4096",
        tm.run(lambda: kernels.gemm_skinny_qkv_rope(pm, x8, Wm, pos8, seq8, tab, bs, c1, None, 0, True, H, G, dim, flag, bias=bias, kv_planes=1,
                                                    n_extra=extra), 3, 10), bytes_=Wm.numel() * 2, like="the one below")
    Wq = rnd((H + 2 * G) * dim, width, scale=0.02)
    inv = torch.tensor([1.0e4 ** (-2.0 * i / dim) for i in range(dim // 2)], dtype=f32, device=dev)
    rec(f"gemm_skinny_qkv_rope (Llama) 8 x {Wq.shape[0]} x 4096",
        tm.run(lambda: kernels.gemm_skinny_qkv_rope(qo, x8, Wq, pos8, seq8, tab, bs, c2, inv, dim, True, H, G, dim, flag), 3, 10), bytes_=Wq.numel() * 2)
    Wu, u8 = rnd(ff, width, scale=0.02), torch.empty(8, ff, dtype=bf, device=dev)
    rec(f"gemm_skinny with relu2: 8 x {ff} x 4096", tm.run(lambda: kernels.gemm_skinny(u8, x8, Wu, act="relu2"), 3, 10), bytes_=Wu.numel() * 2,
        like="the one below")
    rec(f"gemm_skinny (Llama) 8 x {ff} x 4096", tm.run(lambda: kernels.gemm_skinny(u8, x8, Wu), 3, 10), bytes_=Wu.numel() * 2)
    return rows


def kernels_attention(rec, tm, rnd, ints, pos, seq, cu, ctxl, cud, ctxd, flag, T, B, H, G, dim, window):
    """The attention kernels of `kernels_alone` and what stands around them in the latent layer."""
    from lmsf_b200 import kernels
    dev = flag.device
    bf, f32, i32, bs = torch.bfloat16, torch.float32, torch.int32, BLOCK_SIZE
    ones = lambda n: torch.ones(n, device=dev)
    pages = T // bs
    tab = torch.arange(pages, dtype=i32, device=dev).view(1, pages)
    t128 = torch.arange(0, T, 128, dtype=i32, device=dev).flip(0).contiguous()
    t64 = torch.arange(0, T, 64, dtype=i32, device=dev).flip(0).contiguous()
    s128, s64 = torch.zeros_like(t128), torch.zeros_like(t64)
    seen_w, seen_all = sum(min(p + 1, window) for p in range(T)), T * (T + 1) // 2
    fl = lambda seen, hd, h: 4.0 * seen * hd * h
    scale = dim ** -0.5
    dist, one = rnd(H, 257, dtype=f32), torch.zeros(H, device=dev)
    c1, c2 = rnd(pages + 1, 1, G, bs, dim, scale=0.5), rnd(pages + 1, 2, G, bs, dim, scale=0.5)
    q, o = rnd(T, H * dim), torch.empty(T, H * dim, dtype=bf, device=dev)
    own = dict(kv_planes=1, dist=dist, sinks=one)
    tc = lambda c, **ex: tm.run(lambda: kernels.attention_prefill_tc(o, q, c, tab, bs, s128, t128, t128.numel(), cu, ctxl, scale, window, H, G, dim, flag, **ex), 3, 10)
    mma = lambda c, **ex: tm.run(lambda: kernels.attention_prefill(o, q, c, tab, bs, s64, t64, t64.numel(), cu, ctxl, scale, window, H, G, dim, **ex), 3, 10)
    rec(f"attention_prefill_tc, keys that are values, distance table, sink, window {window}: 2048 tokens, 32 heads of 128 over 8", tc(c1, **own),
        flops=fl(seen_w, dim, H), like="the one below")
    rec(f"attention_prefill_tc (keys and values, window {window}) 2048 tokens, 32 heads of 128 over 8", tc(c2), flops=fl(seen_w, dim, H))
    rec(f"attention_prefill (mma.sync), keys that are values, distance table, sink, window {window}: 2048 tokens, 32 heads of 128 over 8", mma(c1, **own),
        flops=fl(seen_w, dim, H), like="the one below")
    rec(f"attention_prefill (mma.sync, keys and values, window {window}) 2048 tokens, 32 heads of 128 over 8", mma(c2), flops=fl(seen_w, dim, H))
    for hd in (256, 128):
        cl, ql, ol = rnd(pages + 1, 1, 1, bs, hd, scale=0.5), rnd(T, H * hd), torch.empty(T, H * hd, dtype=bf, device=dev)
        rec(f"attention_prefill (mma.sync), one cached row of {hd} per token, sinks: 2048 tokens, 32 heads" + ("" if hd == 256 else " (Vufolorn's width)"),
            tm.run(lambda: kernels.attention_prefill(ol, ql, cl, tab, bs, s64, t64, t64.numel(), cu, ctxl, 0.06, 0, H, 1, hd, kv_planes=1, sinks=one), 3, 10),
            flops=fl(seen_all, hd, H), like="the one at 128 below" if hd == 256 else None)
    # ---- decode: 64 requests of 2048 tokens
    pages = B * (CONTEXT // bs)
    tabd = torch.arange(pages, dtype=i32, device=dev).view(B, CONTEXT // bs)

    def decode(planes, n_kv, hd, win, **extras):
        c = rnd(pages, planes, n_kv, bs, hd, scale=0.5)
        qd, od = rnd(B, H * hd), torch.empty(B, H * hd, dtype=bf, device=dev)
        visible = win or CONTEXT
        splits, warps = kernels.decode_plan(B, n_kv, H // n_kv, visible, hd, kernels.decode_widths(hd, H // n_kv))
        need = kernels.attention_decode_scratch_floats(B, H, splits, hd)
        scratch = torch.zeros(max(need, 1), dtype=f32, device=dev)
        sec = tm.run(lambda: kernels.attention_decode(od, qd, c, tabd, bs, None, B, cud, ctxd, scale, win, H, n_kv, hd, splits,
                                                      scratch if need else None, warps, kv_planes=planes, **extras), 3, 10)
        return sec, B * visible * n_kv * hd * 2 * planes

    for name, like, args, ex in (
            (f"attention_decode, keys that are values, distance table, sink, window {window}: 64 requests at 2048, 32 heads of 128 over 8", "the one below",
             (1, G, dim, window), dict(dist=dist, sinks=one)),
            (f"attention_decode (keys and values, window {window}) 64 requests at 2048, 32 heads of 128 over 8", None, (2, G, dim, window), {}),
            ("attention_decode, one cached row of 256 per token, sinks: 64 requests at 2048, 32 heads", "the one below", (1, 1, 256, 0), dict(sinks=one)),
            ("attention_decode (Vufolorn: one cached row of 128) 64 requests at 2048, 32 heads", None, (1, 1, 128, 0), {})):
        sec, nbytes = decode(*args, **ex)
        rec(name, sec, bytes_=nbytes, like=like)
    # ---- the latent layer's small kernels
    rank, rot, q_rank = 192, 64, 1536
    x = rnd(T, q_rank + rank + rot)
    cl, cq = rnd(T // bs + 1, 1, 1, bs, rank + rot), torch.empty(T, q_rank, dtype=bf, device=dev)
    inv = torch.tensor([1.0e4 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=f32, device=dev)
    rec(f"latent_norm_rope_cache_write with the query's vector: ranks {q_rank} and {rank} + {rot} rotated, 2048 tokens",
        tm.run(lambda: kernels.latent_norm_rope_cache_write(x[:, q_rank:], ones(rank), 1e-5, cl, pos, seq, tab, bs, rank, rot, rot, inv, flag,
                                                            interleaved=True, rot_mult=1.2, q_rank=q_rank, wq=ones(q_rank), q_out=cq), 3, 10),
        bytes_=T * (q_rank + rank + rot) * 4, like="the one below")
    xs = rnd(T, rank + rot)
    rec(f"latent_norm_rope_cache_write (Bedenex) rank {rank} + {rot} rotated, 2048 tokens",
        tm.run(lambda: kernels.latent_norm_rope_cache_write(xs, ones(rank), 1e-5, cl, pos, seq, tab, bs, rank, rot, rot, inv, flag), 3, 10),
        bytes_=T * (rank + rot) * 4)
    qh, qa = rnd(T, H * (dim + rot)), torch.empty(T, H * (rank + rot), dtype=bf, device=dev)
    for il in (True, False):
        rec(f"latent_query_rope, {'neighbours' if il else 'halves (Bedenex)'}: 32 heads, {rot} rotated values, 2048 tokens",
            tm.run(lambda: kernels.latent_query_rope(qa, qh, pos, H, dim, rot, rot, inv, rank, rank + rot, interleaved=il), 3, 10),
            bytes_=T * H * rot * 4, like="the one below" if il else None)
    kc = rnd(T, G * dim)
    rec("rope_cache_write of keys alone (no rotation) 2048 x 8 x 128",
        tm.run(lambda: kernels.rope_cache_write(q, kc, None, pos, seq, tab, bs, c1, None, 0, True, H, G, dim, flag), 3, 10), bytes_=T * G * dim * 4,
        like="the one below")
    vc = rnd(T, G * dim)
    rec("rope_cache_write of keys and values (no rotation) 2048 x 8 x 128",
        tm.run(lambda: kernels.rope_cache_write(q, kc, vc, pos, seq, tab, bs, c2, None, 0, True, H, G, dim, flag), 3, 10), bytes_=T * G * dim * 8)


def run(bench, steps, warmup, pk):
    sampler = bench.ClockSampler()
    sampler.start()
    sizes = {}
    for name, cfg in SIZES.items():
        sizes[name] = {"fivedra": measure_model(cfg, [8, 64], steps, warmup, bench),
                       "vufolorn": measure_model(design_bench.SIZES[name][0], [8, 64], steps, warmup, bench),
                       "llama": measure_model(design_bench.SIZES[name][1], [8, 64], steps, warmup, bench)}
    alone = kernels_alone(pk)
    line = {"metric": "prefill and decode tokens/s of the Fivedra design beside the Vufolorn design and the Llama shape of equal width "
                      "(4 layers each, random weights)",
            "unit": "tokens/s", "n_gpus": 1, "steps": steps, "warmup": warmup, "dtype": "bf16", "data": "synthetic",
            "config": {"prefill_tokens": PREFILL_TOKENS, "context": CONTEXT, "block_size": BLOCK_SIZE, "sizes": SIZES,
                       "vufolorn": {k: v[0] for k, v in design_bench.SIZES.items()},
                       "llama": {k: v[1] for k, v in design_bench.SIZES.items()}, "peaks": pk.get("source", "measured")},
            "sizes": sizes, "kernels_alone": alone, "clocks": sampler.stop(), "impl": "ours"}
    print(json.dumps(line))
    return 0
