"""The Fivedra design on the GPU: every mechanism alone against the plain implementation (tests/plain_fivedra.py), then whole
models through the engine's step function in every way of cutting, long decoding, reuse of pages and slots, and generation."""
import math
import random

import numpy as np
import pytest
import torch

import plain_fivedra as P
import traces
import util
from fivedra_configs import BLOCK, CONFIGS, latent, memory, mingru, model, parallel, rotation, window, with_mlp
from test_bedenex_gpu import DEV, F32_TOL, TDT, _context, dev, i32, position_errors, worst_rel, write_model

pytestmark = pytest.mark.gpu
EPS = 1e-5
_folders, _oracles = {}, {}


def folder_of(name, std=None):
    key = (name, std)
    if key not in _folders:
        w = P.random_weights(CONFIGS[name], seed=sum(map(ord, name)), std=std, dtype=torch.bfloat16)
        _folders[key] = (write_model(CONFIGS[name], w, f"lmsf_fiv_{name}_"), w)
    return _folders[key]


def oracle(name, reqs, std=None):
    _, w = folder_of(name, std)
    out = {}
    for rid, toks in reqs.items():
        key = (name, std, tuple(toks))
        if key not in _oracles:
            _oracles[key] = P.forward(CONFIGS[name], w, toks, dtype=torch.float64).float().numpy()
        out[rid] = _oracles[key]
    return out


def requests_for(name, lengths, seed=0):
    return {f"q{i}": util.random_ids(n, CONFIGS[name]["vocab"], seed + 11 * i) for i, n in enumerate(lengths)}


def assert_close(rows, ref, dtype, what):
    """float32: every logit within 3e-5 of the largest.  bfloat16: nothing in this design chooses, so every position holds."""
    if dtype == "float32":
        assert worst_rel(rows, ref) <= F32_TOL, (what, worst_rel(rows, ref))
    else:
        e = position_errors(rows, ref)
        assert e[len(e) // 2] <= 2e-2 and e[-1] <= 6e-2, (what, e[len(e) // 2], e[-1])


# ----------------------------------------------------------------------------- mechanisms alone

def mixer_part(layer, D, W, tdt):
    """The mixer of a layer as the design's description builds it, with weights `W` (names without the layer's prefix)."""
    from lmsf_b200.config.registry import resolve_architecture
    from lmsf_b200.parts.base import build_part, with_nested
    cfg = model(16, D, EPS, 1.0, [with_mlp(layer, None)])
    arch = resolve_architecture(cfg)
    spec = arch.build_spec(arch.parse_config(cfg)).layers[0].parts["mixer"]
    part = build_part("mixer", spec)
    for p, s in with_nested(part, spec):
        get = lambda n: W[n[len("l0.mix."):]].to(tdt)
        p.set_weights({k: dev(torch.cat([get(n) for n in v]) if isinstance(v, list) else get(v)) for k, v in s.weights.items()})
    for p, _ in with_nested(part, spec):
        p.prepare(tdt, torch.device(DEV))
    return part


def mixer_weights(layer, D, seed):
    cfg = model(16, D, EPS, 1.0, [with_mlp(layer, None)])
    return {n: t.float() for n, t in P.sub(P.random_weights(cfg, seed), "l0.mix.").items()}


def double(W):
    return {n: t.double() for n, t in W.items()}


def caches_for(part, bs, pages, slots, tdt):
    from lmsf_b200.parts.base import LayerCache
    c, s = part.cache_spec(), part.state_spec()
    return LayerCache(kv=torch.zeros((pages, c.planes, c.num_kv_heads, bs, c.head_dim), dtype=tdt, device=DEV) if c else None, group=0,
                      state=torch.zeros((slots, *s.shape), dtype=s.dtype, device=DEV) if s else None)


def run_cuts(part, hs, cuts, tdt, bs=16, pages=64):
    """The part's outputs (times what it asks the block for) for sequences hs run side by side: cuts is a list of tuples, how
    many tokens each sequence brings in a step (0: it sits out).  Slots are dealt in another order than the batch's."""
    cache = caches_for(part, bs, pages * len(hs), len(hs) + 2, tdt)
    done, outs = [0] * len(hs), [[] for _ in hs]
    g = torch.Generator().manual_seed(3)
    deal = torch.randperm(pages * len(hs), generator=g).tolist()
    for cut in cuts:
        live = [(s, done[s], n) for s, n in enumerate(cut) if n]
        ctx = _context([(d, n) for _, d, n in live], bs, pages * len(hs), 0, tdt)
        table = ctx.groups[0].block_table
        for row, (s, d, n) in enumerate(live):                              # a sequence keeps its pages over the steps
            used = (d + n + bs - 1) // bs
            table[row, :used] = i32(deal[s * pages:s * pages + used])
        ctx.state_slot = i32([len(hs) - s for s, _, _ in live])
        y = part.forward(ctx, dev(torch.cat([hs[s][d:d + n] for s, d, n in live])), cache).float().cpu() * part.out_scale
        assert int(ctx.error_flag.item()) == 0
        at = 0
        for s, d, n in live:
            outs[s].append(y[at:at + n])
            at += n
            done[s] += n
    assert done == [h.shape[0] for h in hs]
    return [torch.cat(o).double() for o in outs]


def cut_up(lengths, sizes):
    """Steps in which every sequence brings portions of changing size, each from another place of the list."""
    left, steps, j = list(lengths), [], 0
    while any(left):
        cut = tuple(min(l, sizes[(j + 2 * s) % len(sizes)]) for s, l in enumerate(left))
        left = [l - c for l, c in zip(left, cut)]
        steps.append(cut)
        j += 1
    return steps


def every_cut(lengths):
    """Whole; all but the last tokens whole and those one by one; portions of several sizes; pairs of tokens."""
    tail = [min(20, l - 1) for l in lengths]
    ones = [tuple(int(i < t) for t in tail) for i in range(max(tail))]
    return {"whole": [tuple(lengths)], "decode": [tuple(l - t for l, t in zip(lengths, tail))] + ones,
            "portions": cut_up(lengths, [2, 7, 64, 3, 129, 2, 50, 1, 100]), "pairs": cut_up([min(l, 60) for l in lengths], [2]) + cut_up([max(0, l - 60) for l in lengths], [97])}


def check_mixer(layer, D, lengths, dtype, seed, plain, tol=None, bs=16):
    tdt = TDT[dtype]
    g = torch.Generator().manual_seed(seed)
    W = mixer_weights(layer, D, seed)
    hs = [torch.randn(n, D, generator=g).to(tdt) for n in lengths]
    want = [plain(h.double(), double(W)) for h in hs]
    part = mixer_part(layer, D, W, tdt)
    tol = tol or (2e-5 if dtype == "float32" else 3e-2)
    for name, cuts in every_cut(lengths).items():
        for a, b in zip(run_cuts(part, hs, cuts, tdt, bs=bs, pages=2 + max(lengths) // bs), want):
            err = (a - b).abs().max(dim=1).values
            assert float(err.max()) <= tol * float(b.abs().max()), (name, int(err.argmax()), float(err.max() / b.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [50, 37, 96, 8, 260])
def test_min_gru_in_every_cut(width, dtype):
    """One step of the kernel's long form is 256 tokens: a sequence longer than that, one shorter, one of a single token."""
    layer = mingru(width)
    check_mixer(layer, 48, [300, 41, 1], dtype, width, lambda h, W: P.min_gru_mixer(h, W))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_min_gru_keeps_its_state_through_a_thousand_closed_gates(dtype):
    """Gates nearly closed (1 - z close to one) over a long sequence: what the first tokens wrote is still there at the end,
    whole and after portions; 1 - z is not computed as a difference that rounds to one."""
    from lmsf_b200 import kernels
    tdt = TDT[dtype]
    T, w = 1000, 40
    g = torch.Generator().manual_seed(2)
    z = torch.full((T, w), -14.0)
    z[0] = 6.0
    u, gate = torch.randn(T, w, generator=g) * 3, torch.ones(T, w)
    z, u, gate = (x.to(tdt) for x in (z, u, gate))
    a, b = P.sigmoid(-z.double()), P.sigmoid(z.double()) * torch.where(u.double() >= 0, u.double() + 0.5, P.sigmoid(u.double()))
    S, want = torch.zeros(w).double(), []
    for t in range(T):
        S = a[t] * S + b[t]
        want.append(S * P.sigmoid(torch.ones(1).double()))
    want = torch.stack(want)
    p = dev(torch.cat([z, u, gate], 1))
    for cuts in ([T], [1] * 5 + [600, 2, 393], [257, 256, 255, 232]):
        state = torch.zeros(2, w, device=DEV)
        out, done = [], 0
        for n in cuts:
            o = torch.empty(n, w, dtype=tdt, device=DEV)
            x = p[done:done + n]
            kernels.min_gru(o, x[:, :w], x[:, w:2 * w], x[:, 2 * w:], None, None, state, i32([0, n]), i32([1]), 1, n)
            out.append(o.float().cpu().double())
            done += n
        err = float((torch.cat(out) - want).abs().max()) / float(want.abs().max())
        assert err <= (1e-5 if dtype == "float32" else 5e-3), (cuts[:3], err)
        assert float((state[1].cpu().double() - S).abs().max()) <= 1e-5 * float(S.abs().max()) and float(state[0].abs().max()) == 0


def matrix_memory_rows(m, T, seed, tdt, forget=2.0, swing=3.0, dt=torch.float64):
    """Columns q | k | v | i | f of a projection's output and the plain recurrence's outputs (before norm and gate) for them,
    computed in `dt`."""
    H, dk, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    g = torch.Generator().manual_seed(seed)
    p = torch.cat([torch.randn(T, 2 * H * dk + H * dv, generator=g), torch.randn(T, H, generator=g) * swing,
                   torch.randn(T, H, generator=g) * swing + forget], 1).to(tdt)
    x = p.to(dt)
    q = x[:, :H * dk].view(T, H, dk) * dk ** -0.5
    k, v = x[:, H * dk:2 * H * dk].view(T, H, dk), x[:, 2 * H * dk:2 * H * dk + H * dv].view(T, H, dv)
    li, lf = cap * torch.tanh(x[:, -2 * H:-H] / cap), P.log_sigmoid(cap * torch.tanh(x[:, -H:] / cap))
    S, n, top = torch.zeros(H, dk, dv, dtype=dt), torch.zeros(H, dk, dtype=dt), torch.zeros(H, dtype=dt)
    rows = []
    for t in range(T):
        new = torch.maximum(lf[t] + top, li[t])
        a, b = torch.exp(lf[t] + top - new), torch.exp(li[t] - new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        top = new
        rows.append(((S * q[t][:, :, None]).sum(1) / (torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6)[:, None]).flatten())
    return p, torch.stack(rows), (S, n, top)


def run_memory(m, p, cuts, slot_count=3):
    """The kernel over portions `cuts`, chunked from `long` tokens on; returns outputs and the slot's (S, n copies, m copies)."""
    from lmsf_b200 import kernels
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    p = dev(p)
    state = torch.zeros(slot_count, kernels.matrix_memory_state_floats(H, dk, dv), device=DEV)
    zero = torch.zeros(H, device=DEV)
    C = kernels.matrix_memory_chunk_tokens()
    out, done = [], 0
    for n, chunked in cuts:
        x = p[done:done + n]
        o = torch.full((n, H * dv), float("nan"), device=DEV)
        a, b = H * dk, 2 * H * dk + H * dv
        kw = {}
        if chunked:
            items = [(0, c, min(c + C, n), j) for j, c in enumerate(range(0, n, C))]
            kw = dict(items=i32(items), spans=i32([(0, 0, len(items), 0)]), last_chunk=i32([0] * (len(items) - 1) + [1]))
        kernels.matrix_memory(o, x[:, :a], x[:, a:2 * a], x[:, 2 * a:b], x[:, b:b + H], x[:, b + H:b + 2 * H], zero, zero, state,
                              i32([0, n]), i32([1]), 1, H, dk, dv, m["gate_cap"], dk ** -0.5, **kw)
        out.append(o.cpu().double())
        done += n
    tiles = -(-dv // 64)
    s = state[1].cpu().double()
    assert float(state[0].abs().max()) == 0 and float(state[2].abs().max()) == 0
    return torch.cat(out), (s[:H * dk * dv].view(H, dk, dv), s[H * dk * dv:H * dk * (dv + tiles)].view(tiles, H, dk),
                            s[H * dk * (dv + tiles):].view(tiles, H))


SIZES = [memory(2, 48, 64), memory(3, 10, 18, 4.0), memory(1, 33, 70, 9.0), memory(4, 8, 4, 1.5), memory(2, 64, 130, 15.0),
         memory(1, 130, 64, 15.0), memory(1, 256, 100, 15.0), memory(5, 1, 1, 2.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", SIZES, ids=lambda m: "x".join(str(m[k]) for k in ("heads", "dim", "vdim")))
@pytest.mark.parametrize("forget,swing", [(2.0, 3.0), (-3.0, 6.0), (6.0, 12.0)])
def test_matrix_memory_scanned_and_in_chunks_is_the_recurrence(m, dtype, forget, swing):
    """Gates that keep nearly everything, that forget at once, and that sit at their cap; token by token, in chunks, and in
    portions of both kinds; outputs, the state and every tile's copy of n and m."""
    T = 211
    p, want, (S, n, top) = matrix_memory_rows(m, T, 7, TDT[dtype], forget, swing)
    error = lambda x: (x.double() - want).abs() / (1e-5 + want.abs().max(1, keepdim=True).values)
    # the plain recurrence in float32: how far rounding alone moves outputs whose denominator nearly vanishes
    cond = error(matrix_memory_rows(m, T, 7, TDT[dtype], forget, swing, torch.float32)[1])
    for cuts in ([(T, False)], [(T, True)], [(5, False), (64, True), (1, False), (1, False), (140, True)], [(65, True), (63, True), (2, False), (81, True)]):
        got, (s, nn, mm) = run_memory(m, p, cuts)
        err = error(got)
        assert torch.isfinite(got).all() and float(err.max()) <= 1e-4 + 10 * float(cond.max()), (cuts, float(err.max()), float(cond.max()))
        assert float(err.mean()) <= 1e-6 + 3 * float(cond.mean()), (cuts, float(err.mean()), float(cond.mean()))
        assert float((s - S).abs().max()) <= 2e-5 * float(S.abs().max())
        for t in range(nn.shape[0]):
            assert float((nn[t] - n).abs().max()) <= 2e-5 * max(float(n.abs().max()), 1e-6) and float((mm[t] - top).abs().max()) <= 2e-5 * (1 + float(top.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_matrix_memory_returns_what_one_token_wrote_hundreds_before(dtype):
    """One token opens its input gate by far and all others keep theirs shut: a query equal to its key reads its value from any
    place in a chunk, the first and the last of one, and after any cut; forgetting is slow, so the distance shows as well."""
    m = memory(1, 12, 20, 15.0)
    H, dk, dv = 1, 12, 20
    T = 300
    for far in (0, 1, 63, 64, 65, 127, 128, 190, 298):
        g = torch.Generator().manual_seed(far)
        p = torch.cat([torch.randn(T, 2 * dk + dv, generator=g), torch.full((T, 1), -9.0), torch.full((T, 1), 7.0)], 1)
        p[far, -2] = 9.0
        p[far, dk:2 * dk] *= 2.0
        p[T - 1, :dk] = 4.0 * p[far, dk:2 * dk]
        p = p.to(TDT[dtype])
        x = p.double()
        v = x[far, 2 * dk:2 * dk + dv]
        for cuts in ([(T, True)], [(T - 1, True), (1, False)], [(100, True), (199, True), (1, False)], [(T - 20, True), (20, False)]):
            got = run_memory(m, p, cuts)[0][-1]
            assert float((got - v).abs().max()) <= 0.02 * float(v.abs().max()), (far, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,gsize", [(3, 18), (1, 70), (4, 256)])
def test_the_norm_per_head_takes_a_weight_over_all_heads_a_gate_and_a_factor(dtype, heads, gsize):
    from lmsf_b200 import kernels
    g = torch.Generator().manual_seed(gsize)
    tdt, n, V = TDT[dtype], 33, heads * gsize
    x, gate, w = torch.randn(n, V, generator=g) * 5, torch.randn(n, V + 3, generator=g).to(tdt)[:, 3:], torch.randn(V, generator=g)
    buf = torch.zeros(n, V + 8, dtype=tdt, device=DEV)
    kernels.grouped_gated_norm(buf[:, :V], dev(x), dev(gate.contiguous()), dev(w), gsize, EPS, gate_act="sigmoid", out_scale=-1.75)
    want = -1.75 * P.rms(x.double().view(n, heads, gsize), EPS).view(n, V) * w.double() * P.sigmoid(gate.double())
    assert float((buf[:, :V].cpu().double() - want).abs().max()) <= (2e-6 if dtype == "float32" else 5e-3) * float(want.abs().max())
    assert float(buf[:, V:].abs().max()) == 0


# (left, right, left scale, right scale, page size)
PAIRS = [
    (window(4, 2, 24, 0.25, 60, 21), memory(3, 10, 18, 4.0), 0.7, -1.3, 8),
    (window(2, 2, 12, 0.3, 13, 50, 7), memory(1, 33, 70, 9.0), -0.4, 2.0, 16),
    (window(6, 1, 16, 0.4, 200, None, 32), memory(2, 8, 4, 1.5), 1.0, 1.0, 16),
    (window(4, 1, 64, 0.125, 96, 150), memory(2, 64, 130), 0.5, 0.8, 16),
    (window(3, 3, 128, 0.09, 400, 129, 24), memory(4, 24, 64, 2.0), 1.5, 0.3, 32),
    (window(5, 5, 64, 0.1, 20, 7, 6), memory(1, 16, 16, 30.0), 0.0, 1.2, 16),
    (window(2, 1, 144, 0.08, 1000, 64, 2), memory(2, 40, 9), 2.0, 0.0, 16),
    (window(3, 1, 80, 0.1, 50, 1, 40), memory(7, 3, 5), 0.25, 4.0, 16),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("left,right,ls,rs,bs", PAIRS)
def test_two_mixers_side_by_side_in_every_cut(left, right, ls, rs, bs, dtype):
    """Both halves of the pair at once: windows shorter and longer than a page, a tile and where the buckets end, no window, a
    window of one token; factors that are negative, one, zero; three sequences side by side that bring unequal portions."""
    layer = parallel(left, right, ls, rs)
    D, lengths = 56, [231, 77, 1]
    check_mixer(layer, D, lengths, dtype, left["dim"] + right["dim"], lambda h, W: P.parallel_mixer(h, W, layer["mixer"], EPS), bs=bs)


def window_part(m, D, W, tdt, **more):
    from lmsf_b200.parts.attention import PagedAttention
    from lmsf_b200.parts.rope import BucketedDistanceBias
    bias = BucketedDistanceBias(m["heads"], m["bias_max"])
    bias.set_weights({"table": dev(W["rel"].float())})
    part = PagedAttention(D, m["heads"], m["kv_heads"], m["dim"], position_encoding=bias, window=(m.get("mask") or {}).get("size"),
                          scale=m["scale"], bias=True, out_bias=False, values_are_keys=True, unit_sink=True, **more)
    part.set_weights({"qkv": dev(torch.cat([W["q"], W["k"]]), tdt), "qkv_bias": dev(torch.cat([W["q.b"], W["k.b"]]), tdt), "o": dev(W["o"], tdt)})
    part.position_encoding.prepare(tdt, torch.device(DEV))
    part.prepare(tdt, torch.device(DEV))
    return part


def window_weights(g, D, m, scale=1.0):
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    W = {"q": torch.randn(H * d, D, generator=g) * scale / math.sqrt(D), "k": torch.randn(G * d, D, generator=g) / math.sqrt(D),
         "q.b": torch.randn(H * d, generator=g) * 0.5, "k.b": torch.randn(G * d, generator=g) * 0.5,
         "rel": torch.randn(m["buckets"], H, generator=g), "o": torch.randn(D, H * d, generator=g) / math.sqrt(H * d)}
    return {n: t.to(torch.bfloat16).float() for n, t in W.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [64, 128, 48, 160])
def test_every_piece_of_the_window_attention_shows(dim, dtype):
    """Leaving out the one in the denominator, a bias, the table, or shifting the window or a bucket's edge by one moves the
    result by far more than the bound that the part keeps (mistakes planted in the plain implementation)."""
    tdt, D, T = TDT[dtype], 40, 210
    g = torch.Generator().manual_seed(dim)
    m = window(4, 2, dim, 0.6 / math.sqrt(dim), 90, 70, 12)
    W = window_weights(g, D, m)
    h = torch.randn(T, D, generator=g).to(tdt)
    Wd = double(W)
    want = P.window_attention(h.double(), Wd, m)
    tol = 2e-5 if dtype == "float32" else 3e-2
    top = float(want.abs().max())
    got = run_cuts(window_part(m, D, W, tdt), [h], [(T,)], tdt, pages=16)[0]
    assert float((got - want).abs().max()) <= tol * top
    wrong = {"window": dict(m, mask={"size": 69}), "far": dict(m, bias_max=60)}
    others = {n: P.window_attention(h.double(), Wd, mm) for n, mm in wrong.items()}
    for n in ("q.b", "k.b", "rel"):
        others[n] = P.window_attention(h.double(), dict(Wd, **{n: torch.zeros_like(Wd[n])}), m)
    keep = P.softmax_with_sink
    try:
        P.softmax_with_sink = lambda s, seen, sink: keep(s, seen, torch.tensor(-80.0).double())
        others["one"] = P.window_attention(h.double(), Wd, m)
    finally:
        P.softmax_with_sink = keep
    for n, o in others.items():
        assert dtype == "bfloat16" or float((o - want).abs().max()) > 100 * tol * top, n
        assert float((got - want).pow(2).mean().sqrt()) < 0.25 * float((o - want).pow(2).mean().sqrt()), n


def one_key_stands_out(g, m, T, far):
    """A width of twice the head size: the key of a token is the first half of its input, its query the second half (all heads
    alike).  Direction 0 is the far key's alone, and the last query asks for it by far; no other key has a share of it."""
    d, H, G = m["dim"], m["heads"], m["kv_heads"]
    D = 2 * d
    W = window_weights(g, D, m)
    W["q"], W["k"] = torch.zeros(H * d, D), torch.zeros(G * d, D)
    for hd in range(H):
        W["q"][hd * d:(hd + 1) * d, d:] = torch.eye(d)
    for hd in range(G):
        W["k"][hd * d:(hd + 1) * d, :d] = torch.eye(d)
    W["q.b"], W["k.b"] = W["q.b"] * 0, W["k.b"] * 0.2
    W["k.b"].view(G, d)[:, 0] = 0.0
    W["o"] = torch.zeros(D, H * d)
    for hd in range(H):
        W["o"][hd, hd * d] = 1.0                       # what comes out: each head's share of direction 0
    h = torch.randn(T, D, generator=g)
    h[:, 0] = 0.0
    h[:, d:] *= 0.3
    h[far, 0] = 3.0
    h[T - 1, d] = 9.0 / m["scale"] / 3.0
    return W, h, 3.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,size", [(64, 50), (48, 50), (128, 130), (64, 128)])
@pytest.mark.parametrize("back,seen", [(0, True), (1, True), (15, True), (16, True), (17, True), (-2, True), (-1, True), (0, False), (1, False), (17, False)])
def test_a_key_stands_out_just_inside_the_window_and_not_just_outside(dim, size, back, seen, dtype):
    """The key sits on the query itself, next to it, at a page's edge, on the window's oldest position, on the one before that,
    further out; whole, with the last token alone, cut right after the key, and with the last 20 tokens decoded one by one."""
    tdt, T, bs = TDT[dtype], 240, 16
    dist = back if back >= 0 and seen else size + back      # a negative distance counts from the window's edge
    far = T - 1 - dist
    assert (dist < size) == seen
    g = torch.Generator().manual_seed(dim + dist)
    m = window(4, 2, dim, 1.0 / dim, 40, size, 10)
    W, h, big = one_key_stands_out(g, m, T, far)
    h = h.to(tdt)
    want = P.window_attention(h.double(), double(W), m)[T - 1]
    top = float(want.abs().max())
    assert (top > 0.9 * big) == seen and (seen or top < 1e-6)
    part = window_part(m, 2 * dim, W, tdt)
    for cuts in ([T], [T - 1, 1], [far + 1, T - far - 2, 1] if 0 < far < T - 3 else [3, T - 4, 1], [T - 20] + [1] * 20):
        got = run_cuts(part, [h], [(c,) for c in cuts], tdt, bs=bs, pages=16)[0][-1]
        assert float((got - want).abs().max()) <= (2e-5 if dtype == "float32" else 2e-2) * big, (cuts[:3], float((got - want).abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 1, 15, 16, 17, 255, 256, 417])
def test_a_key_far_back_is_found_without_a_window_beyond_the_last_bucket(far, dtype):
    tdt, T, dim = TDT[dtype], 420, 64
    g = torch.Generator().manual_seed(far)
    m = window(2, 1, dim, 1.0 / dim, 100, None, 8)
    W, h, big = one_key_stands_out(g, m, T, far)
    h = h.to(tdt)
    want = P.window_attention(h.double(), double(W), m)[T - 1]
    assert float(want.abs().max()) > 0.8 * big
    part = window_part(m, 2 * dim, W, tdt)
    for cuts in ([T], [T - 1, 1], [far + 1, T - far - 2, 1] if 0 < far < T - 3 else [3, T - 4, 1]):
        got = run_cuts(part, [h], [(c,) for c in cuts], tdt, pages=28)[0][-1]
        assert float((got - want).abs().max()) <= (2e-5 if dtype == "float32" else 2e-2) * big, (cuts, float((got - want).abs().max()))


LATENTS = [latent(3, 20, 12, 14, 40, 28, 0.2, rotation(12, 500.0, (4.0, 40, 4.0, 0.5))),
           latent(2, 16, 4, 40, 16, 8, 0.3, rotation(4, 10000.0)),
           latent(4, 32, 16, 24, 80, 40, 0.15, rotation(16, 2.0e5, (16.0, 128, 16.0, 2.0))),
           latent(1, 8, 6, 12, 130, 50, 0.25, rotation(6, 100.0, (1.0, 64, 2.0, 2.0))),
           latent(5, 64, 64, 64, 192, 100, 0.09, rotation(64, 1.0e4, (40.0, 4096, 32.0, 1.0))),
           latent(2, 24, 16, 16, 300, 20, 0.2, rotation(8, 50.0, (2.0, 32, 8.0, 1.0))),
           latent(2, 128, 64, 32, 512, 24, 0.07, rotation(64, 1.0e4, (8.0, 512, 32.0, 1.0)))]


@pytest.mark.filterwarnings("ignore:kv_rank")
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", LATENTS, ids=lambda l: str(l["mixer"]["kv_rank"]))
def test_latent_attention_with_low_rank_queries_and_stretched_rotation_in_every_cut(layer, dtype):
    """One cached row per token serves every head as key and value; both low-rank vectors are normed; neighbours are rotated by
    stretched angles and stretched in length; ranks inside and beyond the tensor-core kernels."""
    m = layer["mixer"]
    check_mixer(layer, 48, [233, 50, 1], dtype, m["kv_rank"], lambda h, W: P.latent_attention_mixer(h, W, m, EPS))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_piece_of_the_latent_attention_shows(dtype):
    tdt, D, T = TDT[dtype], 48, 230
    layer = latent(3, 8, 16, 20, 48, 24, 0.35, rotation(16, 200.0, (8.0, 64, 8.0, 1.0)))
    m = layer["mixer"]
    g = torch.Generator().manual_seed(5)
    W = mixer_weights(layer, D, 11)
    h = torch.randn(T, D, generator=g).to(tdt)
    Wd = double(W)
    want = P.latent_attention_mixer(h.double(), Wd, m, EPS)
    got = run_cuts(mixer_part(layer, D, W, tdt), [h], [(T - 1,), (1,)], tdt, pages=16)[0]
    rot = m["rot"]
    others = {"unstretched": dict(m, rot=dict(rot, scaling=None)), "ramp": dict(m, rot=dict(rot, scaling=dict(rot["scaling"], fast=2.0))),
              "factor": dict(m, rot=dict(rot, scaling=dict(rot["scaling"], factor=4.0)))}
    outs = {n: P.latent_attention_mixer(h.double(), Wd, mm, EPS) for n, mm in others.items()}
    outs["sink"] = P.latent_attention_mixer(h.double(), dict(Wd, sink=Wd["sink"] * 0 - 40), m, EPS)
    outs["query norm"] = P.latent_attention_mixer(h.double(), dict(Wd, **{"dq.norm": torch.ones_like(Wd["dq.norm"])}), m, EPS)
    outs["key norm"] = P.latent_attention_mixer(h.double(), dict(Wd, **{"dkv.norm": torch.ones_like(Wd["dkv.norm"])}), m, EPS)
    rms = lambda x: float(x.pow(2).mean().sqrt())
    for n, o in outs.items():
        assert rms(got - want) < 0.25 * rms(o - want), (n, rms(got - want), rms(o - want))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 1, 15, 16, 17, 255, 256, 417])
def test_latent_attention_finds_a_key_far_back_at_and_around_page_borders(far, dtype):
    """The stream is [key content | query content | tag]; the key expansion passes the first part of the cached vector and the
    value expansion the tag alone, so among hundreds of keys the last query finds one, whose tag comes out."""
    tdt, T, dk = TDT[dtype], 420, 16
    D, r = 2 * dk + 2, dk + 2
    layer = latent(2, dk, 4, 8, r, dk, 1.0 / dk, rotation(4, 300.0, (4.0, 64, 4.0, 1.0)))
    m = layer["mixer"]
    g = torch.Generator().manual_seed(far)
    W = mixer_weights(layer, D, 3)
    W["dkv"] = torch.zeros(r + 4, D)
    W["dkv"][:dk, :dk], W["dkv"][dk:r, 2 * dk:] = torch.eye(dk), torch.eye(2)
    W["dq"] = torch.zeros(dk, D)
    W["dq"][:, dk:2 * dk] = torch.eye(dk)
    W["dq.norm"], W["dkv.norm"] = torch.ones(dk), torch.ones(r)
    W["uq"] = torch.cat([torch.cat([torch.eye(dk) * 16.0, torch.zeros(4, dk)])] * 2)
    W["uk"] = torch.cat([torch.cat([torch.eye(dk), torch.zeros(dk, 2)], 1)] * 2)
    W["uv"][:, :dk] = 0
    h = torch.randn(T, D, generator=g) * 0.3
    h[:, 0] = h[:, dk] = 0.0
    h[far, :dk] = 0.0
    h[far, 0], h[T - 1, dk] = 4.0, 4.0
    h[T - 1, dk + 1:2 * dk] = 0.0
    h[far, 2 * dk:] = torch.tensor([2.0, -2.0])
    h = h.to(tdt)
    want = P.latent_attention_mixer(h.double(), double(W), m, EPS)[T - 1]
    other = h.clone()
    other[far, 2 * dk:] *= -1
    moved = float((P.latent_attention_mixer(other.double(), double(W), m, EPS)[T - 1] - want).abs().max())
    assert moved > 1.5 * float(want.abs().max())
    part = mixer_part(layer, D, W, tdt)
    for cuts in ([T], [T - 1, 1], [far + 1, T - far - 2, 1] if 0 < far < T - 3 else [3, T - 4, 1]):
        got = run_cuts(part, [h], [(c,) for c in cuts], tdt, pages=28)[0][-1]
        assert float((got - want).abs().max()) <= (5e-5 if dtype == "float32" else 3e-2) * float(want.abs().max()), cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,D,F", [(1, 48, 100), (7, 72, 36), (16, 40, 64), (17, 40, 64), (130, 33, 20)])
def test_squared_relu_feed_forward(n, D, F, dtype):
    """Up to 16 rows the activation is part of the product before it, beyond that a kernel of its own."""
    from lmsf_b200.parts.mlp import PlainMLP
    g, tdt = torch.Generator().manual_seed(n + F), TDT[dtype]
    W = {"up": torch.randn(F, D, generator=g) / math.sqrt(D), "down": torch.randn(D, F, generator=g) / math.sqrt(F)}
    W = {k: v.to(torch.bfloat16).float() for k, v in W.items()}
    h = torch.randn(n, D, generator=g).to(tdt)
    part = PlainMLP(D, F, activation="relu2")
    assert set(part.weight_specs()) == {"up", "down"}
    part.set_weights({k: dev(v, tdt) for k, v in W.items()})
    part.prepare(tdt, torch.device(DEV))
    got = part.forward(None, dev(h)).float().cpu().double()
    want = P.squared_relu_feed_forward(h.double(), double(W))
    assert float((got - want).abs().max()) <= (1e-5 if dtype == "float32" else 2e-2) * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D", [72, 9, 256, 2052])
def test_one_kernel_adds_both_branches_and_applies_both_norms(D, dtype):
    from lmsf_b200 import kernels
    g, tdt, n = torch.Generator().manual_seed(D), TDT[dtype], 21
    res = torch.randn(n, D, generator=g) * 3
    y1, y2 = torch.randn(n, D, generator=g).to(tdt), torch.randn(n, D, generator=g).to(tdt)
    w1, w2 = torch.randn(D, generator=g), torch.randn(D, generator=g)
    for a, b, one, two in ((y1, y2, True, True), (y1, None, True, False), (None, None, True, True), (None, y2, False, True), (y1, y2, False, False)):
        r = dev(res.clone())
        h1 = torch.empty(n, D, dtype=tdt, device=DEV) if one else None
        h2 = torch.empty(n, D, dtype=tdt, device=DEV) if two else None
        kernels.stream_branches(r, dev(a) if a is not None else None, -0.6, dev(b) if b is not None else None, 1.0, h1, dev(w1), h2, dev(w2), EPS)
        x = res.double() + (-0.6 * a.double() if a is not None else 0) + (b.double() if b is not None else 0)
        assert float((r.cpu().double() - x).abs().max()) <= 1e-6 * float(x.abs().max())
        for h, w in ((h1, w1), (h2, w2)):
            if h is not None:
                want = P.zero_centred_norm(x, w.double() - 1, EPS)
                assert float((h.float().cpu().double() - want).abs().max()) <= (2e-6 if dtype == "float32" else 5e-3) * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D", [72, 9])
def test_the_embedding_enters_the_float32_stream_unrounded(D, dtype):
    from lmsf_b200 import kernels
    g = torch.Generator().manual_seed(D)
    table = torch.randn(50, D, generator=g).to(TDT[dtype])
    ids = util.random_ids(33, 50, 1)
    out, flag = torch.empty(33, D, device=DEV), i32([0])
    kernels.embedding_stream(out, dev(table), i32(ids), 9.7, flag)
    assert torch.equal(out.cpu(), table.float()[ids] * torch.tensor(9.7)) and int(flag) == 0
    kernels.embedding_stream(out[:1], dev(table), i32([50]), 1.0, flag)
    assert int(flag) == 1 and float(out[0].abs().max()) == 0


@pytest.mark.parametrize("n", [1, 5, 16, 40])
def test_a_bias_enters_a_product_before_it_is_rounded(n):
    """The sums get the bias in float32 and are rounded once, on the weight-streaming kernel and on the library's product; a
    bias after the rounding is further from the exact result."""
    from lmsf_b200.parts.linear import matmul_tn
    g = torch.Generator().manual_seed(n)
    x, w, b = (torch.randn(*s, generator=g).bfloat16() for s in ((n, 96), (120, 96), (120,)))
    exact = x.double() @ w.double().T + b.double()
    got = matmul_tn(dev(x), dev(w), bias=dev(b)).cpu()
    once = exact.float().bfloat16()
    assert float((got.double() - exact).abs().max()) <= 1.01 * float((once.double() - exact).abs().max()) + 1e-4
    assert float((got == once).float().mean()) > 0.97


# ----------------------------------------------------------------------------- whole models through the step function

def test_the_stream_after_every_layer_is_the_plain_one():
    from lmsf_b200.engine.factory import build_model
    from lmsf_b200.engine.model_runner import ModelRunner, StepEntry
    for name in CONFIGS:
        if name.startswith("R"):
            continue
        folder, w = folder_of(name)
        toks = util.random_ids(67, CONFIGS[name]["vocab"], 4)
        want = []
        P.forward(CONFIGS[name], w, toks, dtype=torch.float64, streams=want)
        net, _, tdt = build_model(folder, "float32", DEV)
        runner = ModelRunner(net, tdt, torch.device(DEV), 8, num_blocks=32, max_num_seqs=2)
        mgr = runner.make_cache_manager()
        got = []
        net.layer_hook = lambda j, x, res: got.append(res.clone())
        mgr.add("a")
        runner.step([StepEntry("a", toks, [])], mgr)
        net.layer_hook = None
        assert len(got) == len(want) == 4
        for j, (a, b) in enumerate(zip(got, want)):
            assert float((a.cpu().double() - b).abs().max()) <= 2e-5 * float(b.abs().max()), (name, j)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["X", "Y", "Z"])
def test_every_way_of_cutting_agrees_with_the_plain_implementation(name, dtype):
    """Whole prompts, prefill then token by token, portions of several sizes down to two tokens, and batches of unequal
    requests with few pages and three live requests (pages and slots are used again)."""
    folder, _ = folder_of(name)
    reqs = requests_for(name, [61, 5, 1, 130, 33, 18, 390 if name == "Z" else 101])
    ref = oracle(name, reqs)
    bs = BLOCK[name]
    modes = {"whole": traces.whole(reqs), "decode": traces.whole(reqs, tail=30), "portions": traces.portions(reqs, [2, 7, 3, 16, 2, 29, 97]),
             "pairs": traces.portions(reqs, [2]), "mixed": traces.mixed(reqs, seed=4, max_live=3, tail=10),
             "mixed with long portions": traces.mixed(reqs, seed=8, max_live=3, sizes=(99, 2, 120, 3), tail=10)}
    got = {}
    for mode, steps in modes.items():
        out = traces.run_inprocess(folder, dtype, steps, bs, traces.max_live_tokens(steps, 64), max_live=3)
        got[mode] = traces.collect(steps, out)
        assert len(got[mode]) == sum(len(t) for t in reqs.values())
        assert_close(got[mode], ref, dtype, mode)
    if dtype == "float32":                            # a position's logits do not depend on the cut beyond rounding
        for mode in modes:
            for key, row in got[mode].items():
                assert np.abs(row - got["whole"][key]).max() <= 3e-5 * np.abs(got["whole"][key]).max(), (mode, key)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_passes_windows_and_pages_and_replays_graphs(dtype):
    """A short prompt, then 150 single tokens: every window passes over decoded tokens, pages behind them are given back; the
    decode steps are replayed from a CUDA graph and must equal the eager steps."""
    from lmsf_b200.engine.factory import build_model
    from lmsf_b200.engine.model_runner import ModelRunner, StepEntry
    folder, _ = folder_of("X")
    reqs = requests_for("X", [160, 158], seed=3)
    ref = oracle("X", reqs)
    net, _, tdt = build_model(folder, dtype, DEV)
    assert all(getattr(p, "graph_safe", False) for p, _ in net.parts_with_specs())
    rows = {}
    for eager in (False, True):
        runner = ModelRunner(net, tdt, torch.device(DEV), 8, num_blocks=48, max_num_seqs=3, enforce_eager=eager)
        mgr = runner.make_cache_manager()
        for rid in reqs:
            mgr.add(rid)
        runner.step([StepEntry(rid, reqs[rid][:8], []) for rid in reqs], mgr)
        got = {rid: [] for rid in reqs}
        for t in range(8, 158):
            lg = runner.step([StepEntry(rid, [reqs[rid][t]], [0]) for rid in reqs], mgr)
            for j, rid in enumerate(reqs):
                got[rid].append(lg[j].float().cpu().numpy())
        assert (len(runner._graphs) > 0) == (not eager)
        tables = [mgr.block_table("q0", g) for g in range(len(runner.storage.groups))]
        assert sum(-1 in t for t in tables) == 2      # both windows have let pages go, the layer without one has not
        rows[eager] = got
        for rid in reqs:
            mgr.free(rid)
    for rid in reqs:
        scale = float(np.abs(ref[rid]).max())
        for i, (a, b) in enumerate(zip(rows[False][rid], rows[True][rid])):
            if dtype == "float32":
                assert np.abs(a - ref[rid][8 + i]).max() <= F32_TOL * scale, (rid, i)
            assert np.abs(a - b).max() <= 1e-5 * scale
    if dtype == "bfloat16":
        assert_close({(rid, 8 + i): a for rid in reqs for i, a in enumerate(rows[False][rid])}, ref, dtype, "decode")


def test_pages_and_slots_of_a_finished_request_serve_the_next():
    """One live request at a time, pages for one and ONE state slot: the second request gets the pages and the states of the
    first, none of which it may see."""
    for name in ("Y", "X"):
        folder, _ = folder_of(name)
        reqs = requests_for(name, [40, 120, 33], seed=9)
        ref = oracle(name, reqs)
        steps = traces.portions(reqs, [13, 2, 98])
        out = traces.run_inprocess(folder, "float32", steps, BLOCK[name], 128, max_live=1)
        assert worst_rel(traces.collect(steps, out), ref) <= F32_TOL


def test_a_request_that_is_dropped_starts_again_from_nothing():
    folder, _ = folder_of("X")
    reqs = requests_for("X", [70, 45], seed=6)
    ref = oracle("X", reqs)
    steps = traces.dropped_and_replayed(reqs, "q0", 31)
    out = traces.run_inprocess(folder, "float32", steps, 8, 2 * traces.max_live_tokens(steps, 64), max_live=2)
    assert worst_rel(traces.collect(steps, out), ref) <= F32_TOL


def test_larger_weights_keep_the_comparison_sharp():
    folder, _ = folder_of("Z", std=0.3)
    reqs = requests_for("Z", [190, 17], seed=5)
    ref = oracle("Z", reqs, std=0.3)
    cond = max(float(np.abs(P.forward(CONFIGS["Z"], folder_of("Z", 0.3)[1], t, dtype=torch.float32).numpy() - ref[r]).max()) for r, t in reqs.items())
    steps = traces.mixed(reqs, seed=1, max_live=2, tail=6)
    out = traces.run_inprocess(folder, "float32", steps, 16, traces.max_live_tokens(steps, 64), max_live=2)
    assert worst_rel(traces.collect(steps, out), ref) <= max(6e-5, 3 * cond / max(float(np.abs(r).max()) for r in ref.values()))


def test_the_trace_program_runs_the_design():
    folder, _ = folder_of("Y")
    reqs = requests_for("Y", [30, 9, 110], seed=2)
    ref = oracle("Y", reqs)
    steps = traces.mixed(reqs, seed=3, max_live=2, tail=4)
    out = traces.run_program(folder, "float32", steps, traces.max_live_tokens(steps, 64))
    assert worst_rel(traces.collect(steps, out), ref) <= F32_TOL


def assert_greedy(cfg, w, prompt, tokens):
    """Every token is the plain implementation's best after those before it (only a near tie may be decided otherwise)."""
    lg = P.forward(cfg, w, list(prompt) + list(tokens), dtype=torch.float64)[len(prompt) - 1:-1]
    for row, got in zip(lg, tokens):
        assert float(row.max() - row[got]) <= 1e-4 * float(row.abs().max())


def test_greedy_generation_through_the_engine():
    """The generation entry point with its scheduler, continuous batching, chunked prompts and sampler."""
    from lmsf_b200 import LLM, SamplingParams
    for name in ("X", "Y"):
        folder, w = folder_of(name)
        cfg = CONFIGS[name]
        prompts = [util.random_ids(n, cfg["vocab"], 50 + i) for i, n in enumerate([23, 4, 141])]
        llm = LLM(folder, dtype="float32", block_size=8, num_gpu_blocks=48, max_num_batched_tokens=110, max_num_seqs=3)
        outs = llm.generate(prompt_token_ids=prompts, sampling_params=SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
        for p, o in zip(prompts, outs):
            assert len(o.outputs[0].token_ids) == 12
            assert_greedy(cfg, w, p, o.outputs[0].token_ids)


def test_preemption_by_recompute_rebuilds_pages_and_state():
    """With few pages the youngest request is dropped and later recomputed from its prompt and its tokens so far: its pages and
    its states start again from nothing.  Greedy and seeded sampling give the tokens of a run with room for all."""
    from lmsf_b200 import LLM, SamplingParams
    folder, _ = folder_of("X")
    cfg = CONFIGS["X"]
    prompts = [util.random_ids(n, cfg["vocab"], 20 + i) for i, n in enumerate([30, 25, 28, 20])]
    sp = [SamplingParams(temperature=0.7 if i % 2 else 0.0, seed=5 + i, max_tokens=40, ignore_eos=True) for i in range(4)]
    roomy = LLM(folder, dtype="float32", block_size=8, num_gpu_blocks=128, max_num_batched_tokens=32, max_num_seqs=4)
    want = [o.outputs[0].token_ids for o in roomy.generate(prompt_token_ids=prompts, sampling_params=sp)]
    assert roomy.engine.scheduler.num_preemptions == 0
    for ahead in (True, False):
        tight = LLM(folder, dtype="float32", block_size=8, num_gpu_blocks=14, max_num_batched_tokens=32, max_num_seqs=4, async_scheduling=ahead)
        got = [o.outputs[0].token_ids for o in tight.generate(prompt_token_ids=prompts, sampling_params=sp)]
        assert tight.engine.scheduler.num_preemptions > 0
        assert got == want, ahead
        tight.engine.cache.check_invariants()
        assert all(tight.engine.cache.num_free_pages(g) == 14 for g in range(len(tight.engine.cache.groups)))


def test_the_example_program_generates_with_the_design():
    """bin/llm_engine_example as a process: a model folder and prompts in, one JSON line per request out."""
    import json
    import os
    import subprocess
    import sys
    folder, w = folder_of("Y")
    cfg = CONFIGS["Y"]
    prompts = [util.random_ids(n, cfg["vocab"], 90 + i) for i, n in enumerate([7, 33])]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cmd = [sys.executable, os.path.join(root, "bin", "llm_engine_example"), "--model", folder, "--dtype", "float32", "--block-size", "16",
           "--num-gpu-blocks", "32", "--max-num-seqs", "4", "--max-num-batched-tokens", "24", "--max-tokens", "8", "--ignore-eos", "--temperature", "0"]
    for p in prompts:
        cmd += ["--prompt-ids", ",".join(str(t) for t in p)]
    proc = subprocess.run(cmd, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True, timeout=300)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [json.loads(ln) for ln in proc.stdout.splitlines() if ln.startswith("{")]
    out = {d["request_id"]: d["token_ids"] for d in lines}
    for i, p in enumerate(prompts):
        assert len(out[i]) == 8
        assert_greedy(cfg, w, p, out[i])


# ----------------------------------------------------------------------------- random configurations

def random_config(seed):
    """Sizes that are no multiples of anything in particular, every optional piece present or absent by chance, values that a
    hand-made configuration tends to make equal or 1."""
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(1, 5)):
        kind = rng.choice(["gru", "pair", "pair", "latent"])
        if kind == "gru":
            layer = mingru(rng.choice([1, 20, 37, 64, 130]))
        elif kind == "pair":
            kv, dim = rng.randint(1, 3), rng.choice([8, 12, 16, 24, 40, 64, 128])
            left = window(kv * rng.randint(1, 3), kv, dim, rng.choice([0.1, 0.3, dim ** -0.5]), rng.choice([17, 50, 128, 1000]),
                          rng.choice([None, 1, 2, 5, 16, 31, 64, 100]), rng.choice([2, 5, 8, 16, 31, 32]))
            right = memory(rng.randint(1, 4), rng.choice([1, 7, 16, 40, 64]), rng.choice([1, 10, 32, 64, 65, 96]), rng.choice([1.0, 5.0, 15.0, 40.0]))
            layer = parallel(left, right, rng.choice([1.0, 0.3, -0.8, 2.0]), rng.choice([1.0, 0.5, -1.2, 1.7]))
        else:
            rot_dim = rng.choice([2, 4, 8, 16, 30])
            layer = latent(rng.randint(1, 5), rng.choice([4, 10, 16, 40]), rot_dim, rng.choice([4, 12, 24, 40]), rng.choice([5, 16, 50, 96, 180]),
                           rng.choice([3, 8, 24, 50]), rng.choice([0.1, 0.3]),
                           rotation(rng.choice([rot_dim, 2]), rng.choice([50.0, 1.0e4, 1.0e6]),
                                    rng.choice([None, (2.0, 32, 4.0, 1.0), (8.0, 64, 8.0, 2.0), (32.0, 1024, 32.0, 1.0), (1.0, 16, 1.0, 1.0)])))
        layers.append(with_mlp(layer, rng.choice([None, 8, 20, 44, 100])))
    return model(rng.choice([61, 128, 257]), rng.choice([36, 50, 56, 72, 104, 140]), rng.choice([1e-6, 1e-5, 1e-3]), rng.choice([1.0, 4.0, 7.3]), layers)


@pytest.mark.parametrize("seed", range(14))
def test_random_configurations(seed):
    name = f"R{seed}"
    CONFIGS[name] = random_config(seed)
    folder, w = folder_of(name)
    rng = random.Random(seed)
    reqs = requests_for(name, [rng.randint(1, 150) for _ in range(4)], seed=seed)
    ref = oracle(name, reqs)
    # how far the plain implementation itself moves when it is run in float32
    scale = max(float(np.abs(r).max()) for r in ref.values())
    cond = max(float(np.abs(P.forward(CONFIGS[name], w, toks, dtype=torch.float32).numpy() - ref[rid]).max()) for rid, toks in reqs.items()) / scale
    bs = rng.choice([8, 16, 32])
    for dtype in ("float32", "bfloat16"):
        for steps in (traces.whole(reqs, tail=5), traces.mixed(reqs, seed=seed, max_live=2, sizes=(7, 2, 100, 3, 29), tail=4)):
            out = traces.run_inprocess(folder, dtype, steps, bs, traces.max_live_tokens(steps, 64), max_live=2)
            rows = traces.collect(steps, out)
            if dtype == "float32":
                assert worst_rel(rows, ref) <= max(5e-5, 3 * cond), (CONFIGS[name], worst_rel(rows, ref), cond)
            else:
                e = position_errors(rows, ref)
                # (a head of one value is divided by its own size: what is left of it, its sign, may turn)
                assert e[len(e) // 2] <= 3e-2 and e[int(0.9 * len(e))] <= 0.1, (CONFIGS[name], e[len(e) // 2], e[int(0.9 * len(e))])
