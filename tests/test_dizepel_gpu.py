"""The Dizepel design on the GPU: every mechanism alone against the plain implementation (tests/plain_dizepel.py), then whole
models through the engine's step function in every way of cutting, long decoding, reuse of pages and slots, and generation."""
import math
import random

import numpy as np
import pytest
import torch

import plain_dizepel as P
import traces
import util
from dizepel_configs import BLOCK, CONFIGS, layer, left, model, right, rotation
from test_bedenex_gpu import DEV, F32_TOL, TDT, _context, dev, i32, position_errors, worst_rel, write_model
from test_fivedra_gpu import double, every_cut, run_cuts

pytestmark = pytest.mark.gpu
EPS = 1e-5
_folders, _oracles = {}, {}


def folder_of(name, std=None):
    key = (name, std)
    if key not in _folders:
        w = P.random_weights(CONFIGS[name], seed=sum(map(ord, name)), std=std, dtype=torch.bfloat16)
        _folders[key] = (write_model(CONFIGS[name], w, f"lmsf_diz_{name}_"), w)
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
    """float32: every logit within 3e-5 of the largest.  bfloat16: a branch that happens to be small at a token is divided by its
    own size, and rounding with it (the plain implementation with its activations rounded moves as far at the same tokens), so
    the bound is on the bulk of the positions."""
    if dtype == "float32":
        assert worst_rel(rows, ref) <= F32_TOL, (what, worst_rel(rows, ref))
    else:
        e = position_errors(rows, ref)
        assert e[len(e) // 2] <= 2e-2 and e[int(0.9 * len(e))] <= 5e-2 and e[-1] <= 0.6, (what, e[len(e) // 2], e[int(0.9 * len(e))], e[-1])


# ----------------------------------------------------------------------------- what lies between two branches

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D", [72, 9, 256, 2052, 4100, 7])
def test_one_kernel_joins_norms_adds_norms_again_and_filters(D, dtype):
    """Every form of the kernel: a branch, a pair, none; norms with and without the mean; a vector; the next norm; the filter."""
    from lmsf_b200 import kernels
    g, tdt, n = torch.Generator().manual_seed(D), TDT[dtype], 13
    rnd = lambda *s: torch.randn(*s, generator=g)
    res = rnd(n, D) * 3 + 5                                  # a mean larger than the deviation
    y1, y2 = (rnd(n, D) * 2 + 1).to(tdt), (rnd(n, D) * 0.1 - 1).to(tdt)
    p1, p2, wp, wn, vec = (rnd(D) for _ in range(5))
    norm = lambda x, w, c: P.centred_norm(x, w, EPS) if c else P.by_rms(x, EPS) * w
    tol = 4e-6 if dtype == "float32" else 6e-3
    for branch, cp, cn, use_vec, taps in (("one", 1, 1, 0, 0), ("pair", 1, 1, 0, 3), (None, 0, 1, 1, 4), ("one", 0, 1, 0, 1), ("pair", 0, 0, 1, 2),
                                          ("one", 1, 0, 1, 9), ("pair", 1, None, 0, 0), (None, 0, 0, 0, 2), ("one", 1, None, 1, 0)):
        r = dev(res.clone())
        h = torch.empty(n, D, dtype=tdt, device=DEV) if cn is not None else None
        x = res.double()
        if branch:
            b = y1.double() if branch == "one" else 0.7 * (P.by_rms(y1.double(), 1e-4) * p1.double() + P.by_rms(y2.double(), 1e-4) * p2.double())
            x = x + norm(b, wp.double(), cp)
        if use_vec:
            x = x + vec.double()
        filt, slots = None, torch.randperm(n + 3, generator=g)[:n]
        if taps:
            f, st = rnd(D, taps), rnd(n + 4, max(1, taps - 1) * D).to(tdt).float()
            state = dev(st.clone())
            filt = (dev(f.t().contiguous()), state, i32(slots.tolist()))
        kernels.stream_layer(r, y=dev(y1) if branch else None, pair=(dev(y2), dev(p1), dev(p2), 1e-4, 0.7) if branch == "pair" else None,
                             w_post=dev(wp), eps_post=EPS, post_centred=bool(cp), vec=dev(vec) if use_vec else None, h=h,
                             w_next=dev(wn) if h is not None else None, eps_next=EPS, next_centred=bool(cn), filt=filt)
        assert float((r.cpu().double() - x).abs().max()) <= 3e-6 * float(x.abs().max()), (branch, cp)
        if h is None:
            continue
        want = norm(x, wn.double(), cn)
        if taps:
            before = st.double()[slots].view(n, -1, D)[:, :taps - 1]
            mine = want[:, None]
            rows = torch.cat([before, mine], 1)                # [n, taps, D], oldest first
            want = want + (rows * f.double().T).sum(1)
            got = state.cpu().double()
            rolled = got[slots].view(n, -1, D)[:, :taps - 1]
            assert float((rolled - rows[:, 1:]).abs().max() if taps > 1 else 0) <= tol * float(rows.abs().max())
            rest = [s for s in range(n + 4) if s not in slots.tolist()]
            assert torch.equal(got[rest], st.double()[rest]) and (taps > 1 or torch.equal(got, st.double()))
        assert float((h.float().cpu().double() - want).abs().max()) <= tol * float(want.abs().max()), (branch, cp, cn, taps)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,taps", [(72, 4), (50, 3), (64, 2), (37, 1), (24, 8), (40, 11), (9, 32)])
def test_the_filter_in_front_of_a_branch_in_every_cut(D, taps, dtype):
    """h + filter(h): whole, portions down to two tokens, single tokens, three sequences side by side; a portion shorter than the
    filter reads inputs of several steps before it."""
    from lmsf_b200.parts.shift import FilterShift
    tdt, g = TDT[dtype], torch.Generator().manual_seed(D)
    part = FilterShift(D, taps)
    f = torch.randn(D, taps, generator=g)
    part.set_weights({"filter": dev(f)})
    part.prepare(tdt, torch.device(DEV))
    lengths = [301, 40, 1]
    hs = [torch.randn(n, D, generator=g).to(tdt) for n in lengths]
    want = [h.double() + P.causal_filter(h.double(), f.double()) for h in hs]

    class AsMixer:
        out_scale = 1.0
        cache_spec = lambda self: None
        state_spec = lambda self: part.state_spec()
        forward = lambda self, ctx, h, cache: part.forward(ctx, h, cache.state)

    for name, cuts in every_cut(lengths).items():
        for a, b in zip(run_cuts(AsMixer(), hs, cuts, tdt), want):
            assert float((a - b).abs().max()) <= (2e-6 if dtype == "float32" else 8e-3) * float(b.abs().max()), name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_step_of_single_tokens_filters_in_the_norm_as_the_filter_alone_does(dtype, monkeypatch):
    """The same decode steps with the filter inside the norm's kernel and as a kernel of its own: the same bits of state, logits
    within rounding."""
    from lmsf_b200.engine.factory import build_model
    from lmsf_b200.engine.model_runner import ModelRunner, StepEntry
    from lmsf_b200.parts import block
    folder, _ = folder_of("X")
    net, _, tdt = build_model(folder, dtype, DEV)
    toks = util.random_ids(30, 211, 8)
    rows = {}
    for fuse in (True, False):
        monkeypatch.setattr(block, "FUSE_NORMS", fuse)
        runner = ModelRunner(net, tdt, torch.device(DEV), 8, num_blocks=16, max_num_seqs=2, enforce_eager=True)
        mgr = runner.make_cache_manager()
        mgr.add("a")
        runner.step([StepEntry("a", toks[:6], [])], mgr)
        rows[fuse] = torch.cat([runner.step([StepEntry("a", [t], [0])], mgr).float().cpu() for t in toks[6:]])
    assert float((rows[True] - rows[False]).abs().max()) <= (1e-6 if dtype == "float32" else 2e-2) * float(rows[True].abs().max())


# ----------------------------------------------------------------------------- the mixers

class Pair:
    """The joined output of a mixer that leaves its two branches to the block."""
    out_scale = 1.0

    def __init__(self, part):
        self.part, self.cache_spec, self.state_spec = part, part.cache_spec, part.state_spec

    def forward(self, ctx, h, cache):
        p = self.part.forward(ctx, h, cache)
        a, b = p.first.double(), p.second.double()
        return p.factor * (P.by_rms(a, p.eps) * p.w_first.double() + P.by_rms(b, p.eps) * p.w_second.double())


def mixer_part(a, b, D, W, tdt):
    """(the pair, its left part, its right part) as the design's description builds them, with weights `W` (mix.* names)."""
    from lmsf_b200.config.registry import resolve_architecture
    from lmsf_b200.parts.base import build_part, with_nested
    cfg = model(16, D, EPS, 1.0, 2, None, [layer(a, b, None)])
    arch = resolve_architecture(cfg)
    spec = arch.build_spec(arch.parse_config(cfg)).layers[0].parts["mixer"]
    part = build_part("mixer", spec)
    for p, s in with_nested(part, spec):
        get = lambda n: W[n[len("l0.mix."):]].to(tdt)
        p.set_weights({k: dev(torch.cat([get(n) for n in v]) if isinstance(v, list) else get(v)) for k, v in s.weights.items()})
    for p, _ in with_nested(part, spec):
        p.prepare(tdt, torch.device(DEV))
    return part, part.left, part.right


def mixer_weights(a, b, D, seed):
    cfg = model(16, D, EPS, 1.0, 2, None, [layer(a, b, None)])
    return {n: t.to(torch.bfloat16).float() for n, t in P.sub(P.random_weights(cfg, seed), "l0.mix.").items()}


def check_cuts(part, hs, want, lengths, tdt, tol, bs=16):
    for name, cuts in every_cut(lengths).items():
        for a, b in zip(run_cuts(part, hs, cuts, tdt, bs=bs, pages=2 + max(lengths) // bs), want):
            err = (a - b).abs().max(dim=1).values
            assert float(err.max()) <= tol * float(b.abs().max()), (name, int(err.argmax()), float(err.max() / b.abs().max()))


ROT = rotation(12, 500.0, (4.0, 40, 4.0, 0.5))
# (left, right, page size): head sizes of every attention kernel, filters of 1 to 11 taps, pairs that 16-byte accesses take and not
MIXERS = [
    (left(4, 2, 24, 0.25, 3, 6.0, ROT), right(6, 10, 12, 3, 2, 5), 8),
    (left(3, 3, 20, 0.3, 4, 30.0, rotation(20, 1.0e4)), right(5, 7, 33, 1, 4, 1), 16),
    (left(6, 1, 12, 0.4, 2, None, rotation(6, 77.0, (8.0, 64, 8.0, 1.0))), right(2, 24, 9, 2, 3, 3), 16),
    (left(5, 1, 16, 0.4, 6), right(3, 8, 20, 3, 1, 4), 16),
    (left(2, 2, 40, 0.2, 1, 3.0), right(4, 16, 5, 2, 5, 2), 32),
    (left(4, 1, 64, 0.2, 4, 12.0, rotation(32, 2.0e5, (16.0, 128, 16.0, 2.0))), right(4, 64, 16, 2, 4, 2), 16),
    (left(3, 3, 128, 0.09, 4, 40.0, rotation(128, 1.0e4)), right(2, 48, 128, 1, 4, 1), 16),
    (left(6, 2, 144, 0.08, 3, 20.0, rotation(16, 900.0)), right(8, 12, 24, 4, 3, 8), 16),
    (left(5, 5, 64, 0.3, 11, 2.0, rotation(64, 50.0, (2.0, 16, 4.0, 1.0))), right(1, 1, 1, 1, 2, 1), 16),
    (left(1, 1, 2, 0.7, 3, 1.0, rotation(2, 9.0)), right(2, 130, 200, 2, 4, 4), 16),
    (left(3, 1, 32, 0.3, 32, 4.0, rotation(16, 60.0)), right(3, 9, 40, 3, 20, 1), 16),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("a,b,bs", MIXERS)
def test_both_halves_and_the_pair_in_every_cut(a, b, bs, dtype):
    """Each half alone (the attention with a state of its own, the state space) and the pair, three sequences side by side that
    bring unequal portions, single tokens beside them, slots and pages dealt in another order."""
    D, lengths = 56, [231, 77, 1]
    tdt, g = TDT[dtype], torch.Generator().manual_seed(a["dim"] + b["vdim"])
    W = mixer_weights(a, b, D, a["dim"])
    hs = [torch.randn(n, D, generator=g).to(tdt) for n in lengths]
    Wd = double(W)
    part, L, R = mixer_part(a, b, D, W, tdt)
    # (a half whose values are few is divided by its own size: bfloat16 moves it by more)
    tol = 3e-5 if dtype == "float32" else 4e-2
    check_cuts(L, hs, [P.attention(h.double(), P.sub(Wd, "left."), a) for h in hs], lengths, tdt, tol, bs)
    check_cuts(R, hs, [P.state_space(h.double(), P.sub(Wd, "right."), b, EPS) for h in hs], lengths, tdt, tol, bs)
    check_cuts(Pair(part), hs, [P.parallel_mixer(h.double(), Wd, {"left": a, "right": b}, EPS) for h in hs], lengths, tdt, 2 * tol, bs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [64, 128, 48, 160])
def test_every_piece_of_the_attention_shows(dim, dtype):
    """Leaving out the sink, the cap, the stretch of frequencies or of lengths, a bias, a tap of a filter, or taking the rotated
    key as the value moves the result by far more than the bound the part keeps (mistakes planted in the plain implementation)."""
    tdt, D, T = TDT[dtype], 40, 210
    g = torch.Generator().manual_seed(dim)
    rot = rotation(dim // 2, 300.0, (4.0, 64, 8.0, 1.0))
    a, b = left(4, 2, dim, 1.2 / math.sqrt(dim), 4, 2.5, rot), right(1, 4, 4, 1, 2, 1)
    W = mixer_weights(a, b, D, dim)
    W["left.sink"] = torch.full((4,), 3.0)
    h = torch.randn(T, D, generator=g).to(tdt)
    Wl = P.sub(double(W), "left.")
    want = P.attention(h.double(), Wl, a)
    L = mixer_part(a, b, D, W, tdt)[1]
    tol = 3e-5 if dtype == "float32" else 3e-2
    got = run_cuts(L, [h], [(T - 1,), (1,)], tdt, pages=16)[0]
    assert float((got - want).abs().max()) <= tol * float(want.abs().max())
    others = {"cap": dict(a, softcap=None), "wider cap": dict(a, softcap=3.0), "frequencies": dict(a, rot=dict(rot, scaling=None)),
              "ramp": dict(a, rot=dict(rot, scaling=dict(rot["scaling"], fast=2.0))), "pairs": dict(a, rot=dict(rot, dims=dim // 2 - 2))}
    outs = {n: P.attention(h.double(), Wl, m) for n, m in others.items()}
    for n, t in (("sink", Wl["sink"] - 60), ("q.b", 0 * Wl["q.b"]), ("k.b", 0 * Wl["k.b"]), ("q.conv", Wl["q.conv"] * torch.tensor([0.0, 1, 1, 1])),
                 ("k.conv", Wl["k.conv"].roll(1, 1))):
        outs[n] = P.attention(h.double(), dict(Wl, **{n: t}), a)
    keep = P.rotary_frequencies
    try:
        P.rotary_frequencies = lambda r: (keep(r)[0], 1.0)
        outs["lengths"] = P.attention(h.double(), Wl, a)
    finally:
        P.rotary_frequencies = keep
    rms = lambda x: float(x.pow(2).mean().sqrt())
    for n, o in outs.items():
        assert rms(got - want) < 0.25 * rms(o - want), (n, rms(got - want), rms(o - want))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_piece_of_the_state_space_shows(dtype):
    tdt, D, T = TDT[dtype], 40, 210
    g = torch.Generator().manual_seed(4)
    a, b = left(1, 1, 16, 0.2, 2), right(6, 16, 24, 3, 4, 2)
    W = mixer_weights(a, b, D, 9)
    h = torch.randn(T, D, generator=g).to(tdt)
    Wr = P.sub(double(W), "right.")
    want = P.state_space(h.double(), Wr, b, EPS)
    got = run_cuts(mixer_part(a, b, D, W, tdt)[2], [h], [(100,), (109,), (1,)], tdt, pages=16)[0]
    outs = {"one group": P.state_space(h.double(), Wr, dict(b, norm_groups=1), EPS)}
    for n, t in (("D", 0 * Wr["D"]), ("conv.b", 0 * Wr["conv.b"]), ("dt_bias", Wr["dt_bias"] + 0.5), ("A_log", Wr["A_log"] + 0.5),
                 ("norm", torch.ones_like(Wr["norm"])), ("conv", Wr["conv"].roll(1, 1))):
        outs[n] = P.state_space(h.double(), dict(Wr, **{n: t}), b, EPS)
    rms = lambda x: float(x.pow(2).mean().sqrt())
    for n, o in outs.items():
        assert rms(got - want) < 0.25 * rms(o - want), (n, rms(got - want), rms(o - want))


def one_key_stands_out(g, a, T, far):
    """A width of twice the head size: a token's key is the first half of its input, its query the second half (all heads alike).
    Direction 0 is the far key's alone, and the last query asks for it by far; nothing is rotated in it, and the filters pass the
    token's own value beside a little of the tokens before."""
    d, H, G, taps = a["dim"], a["heads"], a["kv_heads"], a["conv"]
    D = 2 * d
    n = a["rot"]["dims"]
    at = n                                                # the first direction that passes the rotation unchanged
    W = mixer_weights(a, right(1, 4, 4, 1, 2, 1), D, 7)
    W["left.q"], W["left.k"] = torch.zeros(H * d, D), torch.zeros(G * d, D)
    for hd in range(H):
        W["left.q"][hd * d:(hd + 1) * d, d:] = torch.eye(d)
    for hd in range(G):
        W["left.k"][hd * d:(hd + 1) * d, :d] = torch.eye(d)
    W["left.q.b"] *= 0
    W["left.k.b"] *= 0.1
    W["left.k.b"].view(G, d)[:, at] = 0.0
    for x, heads in (("q", H), ("k", G)):
        W[f"left.{x}.conv"] = torch.full((heads * d, taps), 0.02)
        W[f"left.{x}.conv"][:, -1] = 1.0
    W["left.sink"] = torch.full((H,), -2.0)
    W["left.o"] = torch.zeros(D, H * d)
    for hd in range(H):
        W["left.o"][hd, hd * d + at] = 1.0                # what comes out: each head's share of that direction
    h = torch.randn(T, D, generator=g)
    h[:, at] = 0.0
    h[:, d:] *= 0.2
    h[:, d + at] = 0.0
    h[far, at] = 3.0
    h[T - 1, d + at] = 0.9 * a["softcap"] / a["scale"] / 3.0       # a score near the cap
    W = {k: t.to(torch.bfloat16).float() for k, t in W.items()}
    return W, h, 3.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,far", [(d, f) for d in (64, 128, 48) for f in (0, 1, 15, 16, 17, 127, 128, 255, 256, 402, 417, 418, 419)])
def test_a_key_far_back_is_found_at_and_around_page_and_tile_borders(dim, far, dtype):
    """Whole, with the last token alone, cut right behind the far key, with the last 20 tokens decoded one by one."""
    tdt, T = TDT[dtype], 420
    g = torch.Generator().manual_seed(far)
    a = left(2, 1, dim, 1.0 / dim, 3, 14.0, rotation(dim // 4, 1000.0, (4.0, 64, 8.0, 1.0)))
    W, h, big = one_key_stands_out(g, a, T, far)
    h = h.to(tdt)
    want = P.attention(h.double(), P.sub(double(W), "left."), a)[T - 1]
    assert 0.8 * big < float(want.abs().max()) < 1.2 * big          # the far key takes nearly all of the weight
    L = mixer_part(a, right(1, 4, 4, 1, 2, 1), 2 * dim, W, tdt)[1]
    for cuts in ([T], [T - 1, 1], [far + 1, T - far - 2, 1] if 0 < far < T - 3 else [3, T - 4, 1], [T - 20] + [1] * 20):
        got = run_cuts(L, [h], [(c,) for c in cuts], tdt, pages=28)[0][-1]
        assert float((got - want).abs().max()) <= (3e-5 if dtype == "float32" else 2e-2) * big, (cuts[:3], float((got - want).abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 127, 128, 200, 298])
def test_the_state_space_returns_what_one_token_wrote_hundreds_before(far, dtype):
    """All tokens but one take steps of nearly nothing, so the state neither fades nor takes in; a C equal to the far token's B reads
    its x from any place in a chunk of tokens and after any cut."""
    from lmsf_b200 import kernels
    tdt, T, H, dv, N = TDT[dtype], 300, 2, 20, 12
    g = torch.Generator().manual_seed(far)
    B, C, x = torch.randn(T, N, generator=g), torch.randn(T, N, generator=g), torch.randn(T, H * dv, generator=g)
    dt = torch.full((T, H), -16.0)
    dt[far] = 3.0
    C[T - 1] = 2.0 * B[far] / float(B[far] @ B[far])
    B, C, x, dt = (t.to(tdt) for t in (B, C, x, dt))
    a_log = torch.tensor([-3.0, -6.0])
    step = math.log1p(math.exp(3.0))
    want = step * float(B[far].double() @ C[T - 1].double()) * x[far].double()
    run = scan_runner(H, 1, N, dv, torch.zeros(H), a_log, None, tdt)
    for cuts in ([T], [T - 1, 1], [100, 199, 1], [64, 64, 64, 107, 1], [T - 20] + [1] * 20, [far + 1, T - far - 1]):
        got = run(C, B, x, dt, cuts)[0][-1]
        assert float((got - want).abs().max()) <= 0.01 * float(want.abs().max()), (cuts[:3], got[:3], want[:3])


def scan_runner(H, G, N, dv, dt_bias, a_log, skip, tdt):
    """run(q, k, v, dt, cuts) -> (outputs, the slot's state [H, dv, N]) of the scan as the mixer launches it."""
    from lmsf_b200.parts.recurrent import SelectiveStateSpace
    part = SelectiveStateSpace(8, H, dv, N, G, 1, 1, EPS)
    part._f32 = {"dt_bias": dev(dt_bias.float()), "a_log": dev(a_log.float()), "skip": dev(skip.float()) if skip is not None else torch.zeros(H, device=DEV)}

    def run(q, k, v, dt, cuts):
        state = torch.zeros(3, part.state_floats(), device=DEV)
        out, done = [], 0
        for n in cuts:
            ctx = _context([(done, n)], 16, 64, 0, tdt)
            ctx.state_slot = i32([1])
            y = torch.full((n, H * dv), float("nan"), device=DEV)
            part.scan(ctx, *(dev(t[done:done + n].contiguous()) for t in (q, k, v, dt)), state, y)
            out.append(y.cpu().double())
            done += n
        assert float(state[0].abs().max()) == 0 and float(state[2].abs().max()) == 0
        return torch.cat(out), state[1, :part.matrix_floats].cpu().double().view(H, dv, N)

    return run


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,N,dv", [(4, 2, 16, 24), (2, 1, 128, 64), (6, 3, 7, 5), (1, 1, 1, 1), (3, 1, 200, 130), (8, 2, 64, 48), (2, 2, 256, 40)])
@pytest.mark.parametrize("fade", [-6.0, 0.0, 3.0])
def test_the_scan_in_chunks_and_token_by_token_is_the_recurrence(H, G, N, dv, fade, dtype):
    """States that hardly fade, fade within a chunk, and fade at once (a chunk's decays fall below what float32 holds); outputs and
    the state left behind; whole, in portions of both kinds, token by token."""
    T, tdt = 211, TDT[dtype]
    g = torch.Generator().manual_seed(H * 100 + N)
    q, k, v = (torch.randn(T, w, generator=g).to(tdt) for w in (G * N, G * N, H * dv))
    dt = torch.randn(T, H, generator=g).to(tdt)
    dt_bias, a_log, skip = torch.randn(H, generator=g), torch.randn(H, generator=g) + fade, torch.randn(H, generator=g)
    step = torch.nn.functional.softplus(dt.double() + dt_bias.double(), threshold=1e9)
    decay = torch.exp(-torch.exp(a_log.double()) * step)
    S, want = torch.zeros(H, dv, N).double(), []
    heads = lambda t: t.double().view(T, G, N).repeat_interleave(H // G, 1)
    for t in range(T):
        S = decay[t][:, None, None] * S + step[t][:, None, None] * v.double().view(T, H, dv)[t][:, :, None] * heads(k)[t][:, None, :]
        want.append(((S * heads(q)[t][:, None, :]).sum(-1) + skip.double()[:, None] * v.double().view(T, H, dv)[t]).flatten())
    want = torch.stack(want)
    run = scan_runner(H, G, N, dv, dt_bias, a_log, skip, tdt)
    scale = want.abs().max(1, keepdim=True).values.clamp(min=float(want.abs().max()) * 1e-2)
    for cuts in ([T], [5, 64, 1, 1, 140], [65, 63, 2, 81], [128, 83], [1] * 3 + [200] + [2] * 4):
        got, s = run(q, k, v, dt, cuts)
        assert torch.isfinite(got).all()
        assert float(((got - want).abs() / scale).max()) <= 2e-5, (cuts, float(((got - want).abs() / scale).max()))
        assert float((s - S).abs().max()) <= 1e-5 * float(S.abs().max()), cuts


# ----------------------------------------------------------------------------- capped scores in every attention kernel

@pytest.mark.parametrize("hd", [16, 64, 80, 128, 160, 256])
@pytest.mark.parametrize("size,cap", [(0.2, 50.0), (3.0, 5.0), (40.0, 20.0)])
@pytest.mark.parametrize("H,G,window", [(4, 2, 0), (3, 1, 40), (2, 2, 0)])
def test_capped_scores_in_every_kernel(hd, size, cap, H, G, window):
    """Scores far below the cap (the series), around it, far beyond it (flat): single tokens, portions on both prefill kernels, a
    batch of unequal requests, with a sink, beside the generic kernel; a cap left out shows."""
    from lmsf_b200 import kernels
    from lmsf_b200.parts.attention import paged_attend
    from lmsf_b200.parts import attention as att
    bs, tdt = 16, torch.bfloat16
    seqs = [(150, 1), (0, 140), (33, 70), (7, 1), (300, 2)]
    ctx = _context(seqs, bs, 80, 3, tdt)
    g = torch.Generator().manual_seed(hd)
    n = ctx.n_tokens
    cache = torch.randn(80, 2, G, bs, hd, generator=g).to(tdt)
    q = (torch.randn(n, H * hd, generator=g) * size).to(tdt)
    sinks = torch.randn(H, generator=g)
    scale = 1.0 / math.sqrt(hd)
    table = ctx.groups[0].block_table.cpu()

    def plain(cap_):
        out = torch.zeros(n, H, hd).double()
        row = 0
        for s, (a, b) in enumerate(seqs):
            keys = torch.stack([cache[table[s, p // bs], :, :, p % bs] for p in range(a + b)]).double()     # [T, 2, G, hd]
            for i in range(b):
                pos = a + i
                lo = max(0, pos - window + 1) if window else 0
                for h in range(H):
                    kk, vv = keys[lo:pos + 1, 0, h // (H // G)], keys[lo:pos + 1, 1, h // (H // G)]
                    sc = P.cap_scores((kk @ q[row].double().view(H, hd)[h]) * scale, cap_)
                    e = torch.exp(sc - torch.maximum(sc.max(), sinks[h].double()))
                    out[row, h] = (e @ vv) / (e.sum() + torch.exp(sinks[h].double() - torch.maximum(sc.max(), sinks[h].double())))
                row += 1
        return out.view(n, H * hd)

    want, uncapped = plain(cap), plain(None)
    kv, qd, got = dev(cache), dev(q), {}
    for name, tc, generic in (("tcgen05", True, False), ("mma", False, False), ("generic", False, True)):
        keep, att.USE_TC_PREFILL = att.USE_TC_PREFILL, tc
        try:
            out = torch.full((n, H * hd), float("nan"), dtype=tdt, device=DEV)
            ctx.extras.clear()
            if generic:
                ctx.extras["force_generic_attention"] = True
            paged_attend(ctx, out, qd, kv, ctx.groups[0], num_heads=H, num_kv_heads=G, head_dim=hd, scale=scale, window=window or None,
                         softcap=cap, sinks=dev(sinks))
        finally:
            att.USE_TC_PREFILL = keep
        got[name] = out.cpu().double()
        err = float((got[name] - want).abs().max())
        assert err <= 1.5e-2 * float(want.abs().max()), (name, err)
    assert int(ctx.error_flag.item()) == 0
    if size > 1:
        assert float((uncapped - want).abs().mean()) > 5 * float((got["tcgen05"] - want).abs().mean())
    assert kernels.mma_attention_supported(tdt, hd)


# ----------------------------------------------------------------------------- whole models through the step function

def test_the_stream_after_every_layer_run_is_the_plain_one():
    from lmsf_b200.engine.factory import build_model
    from lmsf_b200.engine.model_runner import ModelRunner, StepEntry
    for name in ("X", "Y", "Z"):
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
        assert len(got) == len(want) == len(P.layer_runs(CONFIGS[name]))
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
def test_a_batch_of_unequal_requests_gives_what_each_gives_alone(dtype):
    """One step that holds a long portion, a pair, single tokens and a request's first token, beside each of them alone."""
    folder, _ = folder_of("Z")
    reqs = requests_for("Z", [140, 12, 31, 9], seed=7)
    cut = {"q0": 130, "q1": 10, "q2": 30, "q3": 8}
    alone = {}
    for rid, toks in reqs.items():
        steps = [{"step": 0, "entries": [{"id": rid, "tokens": toks[:cut[rid]], "want": []}], "end": []},
                 {"step": 1, "entries": [{"id": rid, "tokens": toks[cut[rid]:], "want": list(range(len(toks) - cut[rid]))}], "end": [rid]}]
        alone.update(traces.collect(steps, traces.run_inprocess(folder, dtype, steps, 16, 256, max_live=4)))
    first = [{"id": r, "tokens": t[:cut[r]], "want": []} for r, t in reqs.items()]
    rest = [{"id": r, "tokens": t[cut[r]:], "want": list(range(len(t) - cut[r]))} for r, t in reqs.items()]
    steps = [{"step": 0, "entries": first, "end": []}, {"step": 1, "entries": rest[::-1], "end": list(reqs)}]
    together = traces.collect(steps, traces.run_inprocess(folder, dtype, steps, 16, 512, max_live=4))
    assert set(together) == set(alone)
    for k, row in together.items():
        assert np.abs(row - alone[k]).max() <= (2e-6 if dtype == "float32" else 3e-2) * np.abs(alone[k]).max(), k


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_passes_pages_and_replays_graphs(dtype):
    """A prompt of two tokens, then 150 single tokens; the decode steps are replayed from a CUDA graph and must equal the eager
    steps (in bfloat16 the graph's padding changes nothing either)."""
    from lmsf_b200.engine.factory import build_model
    from lmsf_b200.engine.model_runner import ModelRunner, StepEntry
    folder, _ = folder_of("X")
    reqs = requests_for("X", [160, 158, 155], seed=3)
    ref = oracle("X", reqs)
    net, _, tdt = build_model(folder, dtype, DEV)
    assert all(getattr(p, "graph_safe", False) for p, _ in net.parts_with_specs())
    rows = {}
    for eager in (False, True):
        runner = ModelRunner(net, tdt, torch.device(DEV), 8, num_blocks=64, max_num_seqs=3, enforce_eager=eager)
        mgr = runner.make_cache_manager()
        for rid in reqs:
            mgr.add(rid)
        runner.step([StepEntry(rid, reqs[rid][:2], []) for rid in reqs], mgr)
        got = {rid: [] for rid in reqs}
        for t in range(2, 152):
            lg = runner.step([StepEntry(rid, [reqs[rid][t]], [0]) for rid in reqs], mgr)
            for j, rid in enumerate(reqs):
                got[rid].append(lg[j].float().cpu().numpy())
        assert (len(runner._graphs) > 0) == (not eager)
        rows[eager] = got
        for rid in reqs:
            mgr.free(rid)
    for rid in reqs:
        scale = float(np.abs(ref[rid]).max())
        for i, (a, b) in enumerate(zip(rows[False][rid], rows[True][rid])):
            if dtype == "float32":
                assert np.abs(a - ref[rid][2 + i]).max() <= F32_TOL * scale, (rid, i)
            assert np.abs(a - b).max() <= (1e-5 if dtype == "float32" else 2e-2) * scale
    if dtype == "bfloat16":
        assert_close({(rid, 2 + i): a for rid in reqs for i, a in enumerate(rows[False][rid])}, ref, dtype, "decode")


def test_pages_and_slots_of_a_finished_request_serve_the_next():
    """One live request at a time, pages for one and ONE state slot: the second request gets the pages and the states of the
    first, none of which it may see."""
    for name in ("Y", "X"):
        folder, _ = folder_of(name)
        reqs = requests_for(name, [40, 120, 1, 33], seed=9)
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
    for _ in range(rng.randint(1, 4)):
        kv, dim = rng.randint(1, 3), rng.choice([8, 12, 16, 24, 40, 64, 128])
        rot = None
        if rng.random() < 0.8:
            rot = rotation(rng.choice([2, dim // 2 // 2 * 2, dim]), rng.choice([50.0, 1.0e4, 1.0e6]),
                           rng.choice([None, (2.0, 32, 4.0, 1.0), (8.0, 64, 8.0, 2.0), (32.0, 1024, 32.0, 1.0), (1.0, 16, 1.0, 1.0)]))
        a = left(kv * rng.randint(1, 3), kv, dim, rng.choice([0.1, 0.3, dim ** -0.5]), rng.choice([1, 2, 3, 4, 4, 5, 7]),
                 rng.choice([None, 2.0, 15.0, 50.0]), rot)
        groups = rng.randint(1, 3)
        heads, vdim = groups * rng.randint(1, 3), rng.choice([4, 8, 10, 24, 64])
        parts = rng.choice([p for p in range(1, 9) if heads * vdim % p == 0 and heads * vdim // p > 3])
        b = right(heads, vdim, rng.choice([1, 5, 16, 40, 64, 130]), groups, rng.choice([1, 2, 3, 4, 4, 6]), parts)
        layers.append(layer(a, b, rng.choice([None, 8, 20, 44, 100])))
    n = len(layers)
    start = rng.randint(0, n - 1)
    loop = rng.choice([None, (start, rng.randint(start, n), rng.randint(1, 3))])
    return model(rng.choice([61, 128, 257]), rng.choice([36, 50, 56, 72, 104, 140]), rng.choice([1e-6, 1e-5, 1e-3]), rng.choice([1.0, 4.0, 7.3]),
                 rng.choice([1, 2, 3, 4, 5]), loop, layers)


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
                assert e[len(e) // 2] <= 4e-2 and e[int(0.9 * len(e))] <= 0.12, (CONFIGS[name], e[len(e) // 2], e[int(0.9 * len(e))])
