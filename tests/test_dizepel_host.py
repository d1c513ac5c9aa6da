"""Host side of the Dizepel design: its configuration, its description as data, its tensor names, and the identities that the
engine's kernels rest on, checked on the plain implementation alone."""
import copy
import json
import math

import pytest
import torch

import plain_dizepel as P
from dizepel_configs import CONFIGS, left, right

CFG = CONFIGS["X"]


def build(cfg):
    from lmsf_b200.config.registry import resolve_architecture
    from lmsf_b200.parts.decoder import DecoderModel
    arch = resolve_architecture(cfg)
    typed = arch.parse_config(cfg)
    return typed, DecoderModel(arch.build_spec(typed))


def test_the_design_is_found_by_its_name_and_described_as_data():
    from lmsf_b200.cache.storage import plan_groups
    typed, model = build(CFG)
    assert typed.canon_taps == 4 and typed.embed_scale == 3.0 and (typed.loop_start, typed.loop_stop, typed.loop_times) == (1, 3, 3)
    # the span is unrolled; every run of a layer has a cache and states of its own
    assert [(c.layer, c.entry, c.entry_pass) for c in model.calls] == \
        [(0, None, 0), (1, 0, 0), (2, None, 0), (1, 0, 1), (2, None, 0), (1, 0, 2), (2, None, 0)]
    groups, _ = plan_groups(model)
    # keys and values are cached apart although one projection makes both (heads padded to multiples of 16)
    assert {tuple(g.calls): (g.spec.num_kv_heads, g.spec.head_dim, g.spec.planes, g.spec.window) for g in groups} == \
        {(0,): (2, 32, 2, None), (1, 3, 5): (3, 32, 2, None), (2, 4, 6): (1, 16, 2, None)}
    up4 = lambda n: (n + 3) // 4 * 4
    want = [(6 * 10 * 12 + 1 * (60 + 2 * 36), 2 * (4 + 2) * 32), (5 * 7 * 33 + 3 * (35 + 66), 3 * 6 * 32), (2 * 24 * 9 + 2 * (48 + 36), 1 * 7 * 16)]
    for j, c in enumerate(model.calls):
        a, b = want[c.layer]
        assert model.call_state_spec(j).shape == (up4(up4(a) + b),)
        extra = model.call_extra_state_specs(j)
        assert {r: s.shape for r, s in extra.items()} == {r: (3 * 72,) for r in (("mixer_shift",) if c.layer == 1 else ("mixer_shift", "ffn_shift"))}
    assert model.blocks[1].feed_forward is None and model.blocks[1].ffn_shift is None
    assert all(getattr(p, "graph_safe", False) for p, _ in model.parts_with_specs())
    assert all(b.mixer_norm.centred and b.mixer_post.centred for b in model.blocks) and model.final_norm.centred


def test_tensor_names_and_shapes_are_those_of_the_design():
    from lmsf_b200.weights.loader import collect_requirements
    for name, cfg in CONFIGS.items():
        _, model = build(cfg)
        want = {k: tuple(v) for k, v in P.tensor_shapes(cfg).items()}
        asked = set()
        for _, _, wspec, names in collect_requirements(model):
            for i, n in enumerate(names):
                asked.add(n)
                assert wspec.matches(i, want[n]), n
        assert asked == set(want), (name, asked ^ set(want))


def test_a_span_of_no_layers_is_no_span():
    cfg = copy.deepcopy(CFG)
    cfg["loop"] = {"start": 2, "stop": 2, "times": 5}
    typed, model = build(cfg)
    assert not typed.has_loop and [c.layer for c in model.calls] == [0, 1, 2] and P.layer_runs(cfg) == [(0, None), (1, None), (2, None)]
    for loop, runs in (((0, 3, 1), [0, 1, 2]), ((0, 1, 4), [0, 0, 0, 0, 1, 2]), ((2, 3, 2), [0, 1, 2, 2])):
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
        _, model = build(cfg)
        assert [c.layer for c in model.calls] == runs == [i for i, _ in P.layer_runs(cfg)]
        assert [c.entry_pass for c in model.calls if c.entry is not None] == list(range(loop[2]))


@pytest.mark.parametrize("change,needle", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=48), "values that are the keys"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=4), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "ff"),
    (lambda c: c["canon"].pop("taps"), "taps"),
    (lambda c: c["loop"].update(stop=4), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].update(eps=0), "eps"),
])
def test_a_configuration_that_does_not_fit_is_refused_with_its_key(change, needle):
    from lmsf_b200.config import ConfigError
    cfg = copy.deepcopy(CFG)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        build(cfg)
    assert needle in str(e.value)


def test_missing_and_misshapen_tensors_are_reported_together(tmp_path):
    from lmsf_b200.weights.loader import WeightError, check_tensors
    from lmsf_b200.weights.safetensors_io import open_model_tensors, write_safetensors
    _, model = build(CFG)
    w = P.random_weights(CFG, 0)
    del w["l2.mix.left.sink"]
    w["l0.mix.left.k.conv"] = torch.ones(48, 4, dtype=torch.bfloat16)
    w["l9.extra"] = torch.ones(2, dtype=torch.bfloat16)
    w["l1.norm2"] = torch.ones(72, dtype=torch.bfloat16)                 # layer 1 has no feed-forward: its norm may be stored
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    write_safetensors(str(tmp_path / "model.safetensors"), [(n, t.dtype, tuple(t.shape)) for n, t in w.items()], lambda n: w[n])
    with pytest.raises(WeightError) as e:
        check_tensors(model, open_model_tensors(str(tmp_path)), str(tmp_path))
    assert e.value.missing == ["l2.mix.left.sink"] and e.value.unexpected == ["l9.extra"]
    assert [x[0] for x in e.value.wrong_shape] == ["l0.mix.left.k.conv"]


def test_blocks_that_only_divide_refuse_a_norm_that_takes_the_mean_off():
    from lmsf_b200.parts.base import LayerSpec, PartSpec
    from lmsf_b200.parts.decoder import DecoderModel
    _, model = build(CFG)
    norm = PartSpec("layernorm", dict(hidden_size=72, eps=1e-5), {"weight": "n"})
    mixer = PartSpec("min_gru", dict(hidden_size=72, width=8), {"zxg": ["z", "x", "g"], "z_bias": "zb", "x_bias": "xb", "o": "o"})
    spec = copy.copy(model.spec)
    spec.order = model.spec.order[:1]
    for block, parts in (("branch_norm", {"mixer": mixer, "mixer_post_norm": norm}), ("parallel_norms", {"mixer_norm": norm, "mixer": mixer}),
                         ("parallel_gated", {"norm": norm, "mixer": mixer, "gates": PartSpec("gate_logits", dict(in_features=72, out_features=72), {"weight": "w", "bias": "b"})})):
        spec.layers = [LayerSpec(block, parts)]
        with pytest.raises(ValueError, match="rmsnorm"):
            DecoderModel(spec)
    spec.layers = [LayerSpec("pre_norm", {"mixer_norm": norm, "mixer": model.spec.layers[0].parts["mixer"], "ffn_norm": norm,
                                          "feed_forward": model.spec.layers[0].parts["feed_forward"]})]
    with pytest.raises(ValueError, match="pair"):
        DecoderModel(spec)


def test_a_stretching_rotation_and_an_odd_pair_of_mixers_are_refused():
    from lmsf_b200.parts.attention import PagedAttention
    with pytest.raises(ValueError, match="values that are the keys"):
        PagedAttention(32, 2, 1, 16, qk_filter=4)
    with pytest.raises(ValueError, match="sink"):
        PagedAttention(32, 2, 1, 16, learned_sink=True, unit_sink=True)
    from lmsf_b200.parts.parallel_mixers import NormedParallelMixers
    from lmsf_b200.parts.recurrent import SelectiveStateSpace
    space = SelectiveStateSpace(32, 2, 8, 4, 1, 4, 1, 1e-5)
    with pytest.raises(ValueError, match="side by side"):
        NormedParallelMixers(PagedAttention(32, 2, 1, 16, values_are_keys=True), space, 1e-5)


def test_head_weights_are_padded_with_their_filters():
    """Heads of 20 values are kept 32 wide: rows of the matrix, of the bias and of the filter move together."""
    from lmsf_b200.parts.attention import PagedAttention
    part = PagedAttention(8, 3, 1, 20, bias=True, out_bias=False, values_are_keys=True, qk_filter=3, learned_sink=True)
    g = torch.Generator().manual_seed(0)
    t = {n: torch.randn(*s, generator=g) for n, s in dict(qkv=(80, 8), qkv_bias=(80,), qk_filter=(80, 3), o=(8, 60), sink=(3,)).items()}
    part.set_weights(dict(t))
    for n in ("qkv", "qkv_bias", "qk_filter"):
        got = getattr(part, n).reshape(4, 32, -1)
        assert torch.equal(got[:, :20].flatten(), t[n].flatten()) and float(got[:, 20:].abs().max()) == 0
    assert torch.equal(part.o.reshape(8, 3, 32)[:, :, :20].flatten(), t["o"].flatten())
    assert part.kv_planes == 2 and part.filter_state_floats() == 2 * 4 * 32


# ----------------------------------------------------------------------------- identities

def test_the_polynomial_of_the_hyperbolic_tangent_in_the_kernels_header_meets_it():
    """The ten coefficients in attention_mma.cuh are the interpolation of tanh(x) / x in u = x^2 at the Chebyshev points of [0, 1.5^2];
    evaluated in float32 they give the quotient within float32's rounding."""
    import os
    import re
    import numpy as np
    from lmsf_b200.csrc import build
    text = open(os.path.join(build.CSRC_DIR, "attention_mma.cuh")).read()
    body = re.search(r"c\[kTanhTerms\] = \{([^}]*)\}", text).group(1)
    coef = [float(x.strip().rstrip("f")) for x in body.replace("\n", " ").split(",")]
    assert len(coef) == 10 and float(re.search(r"kTanhFar = ([0-9.]+)f", text).group(1)) == 1.5
    f = lambda u: np.tanh(np.sqrt(u)) / np.sqrt(u)
    want = np.polynomial.Chebyshev.interpolate(f, 9, domain=[0, 2.25]).convert(kind=np.polynomial.Polynomial).coef
    assert np.allclose(coef, want, rtol=1e-7, atol=1e-12)
    u = np.linspace(1e-9, 2.25, 50001).astype(np.float32)
    p = np.full_like(u, np.float32(coef[-1]))
    for c in coef[-2::-1]:
        p = (p.astype(np.float64) * u + np.float32(c)).astype(np.float32)
    assert float(np.abs(p / f(u.astype(np.float64)) - 1).max()) < 2.5e-7


def test_the_series_of_the_hyperbolic_tangent_is_close_where_it_is_used():
    """x (1 + u (-1/3 + u (2/15 + u (-17/315 + u 62/2835)))), u = x^2: within 1e-8 of tanh relative to it up to 1/4."""
    x = torch.linspace(1e-4, 0.25, 5001).double()
    u = x * x
    t = x * (1 + u * (-1 / 3 + u * (2 / 15 + u * (-17 / 315 + u * 62 / 2835))))
    assert float(((t - torch.tanh(x)) / torch.tanh(x)).abs().max()) < 1e-8
    big = torch.linspace(0.25, 60.0, 2001).double()
    assert torch.allclose(1 - 2 / (1 + torch.exp(2 * big)), torch.tanh(big), rtol=1e-12)


def test_chunks_of_the_state_space_equal_the_recurrence():
    """With F the sum of log decays since a chunk's start: what a chunk adds to the state is sum_s exp(F_end - F_s) step_s B_s x_s^T,
    and a token reads exp(F_t) S_before^T C_t + sum_{s <= t} exp(F_t - F_s) step_s (B_s . C_t) x_s."""
    m = right(3, 5, 7, 1, 3, 1)
    g = torch.Generator().manual_seed(1)
    T, H, dv, N = 41, 3, 5, 7
    x, B, C = torch.randn(T, H, dv, generator=g).double(), torch.randn(T, N, generator=g).double(), torch.randn(T, N, generator=g).double()
    step, rate = torch.rand(T, H, generator=g).double() * 2, torch.rand(H, generator=g).double() * 3
    S, want = torch.zeros(H, N, dv).double(), []
    for t in range(T):
        S = torch.exp(-rate * step[t])[:, None, None] * S + step[t][:, None, None] * B[t][None, :, None] * x[t][:, None, :]
        want.append((S * C[t][None, :, None]).sum(1))
    S, got = torch.zeros(H, N, dv).double(), []
    for a in range(0, T, 8):
        b = min(a + 8, T)
        F = torch.cumsum(-rate * step[a:b], 0)
        for t in range(b - a):
            y = torch.exp(F[t])[:, None] * (S * C[a + t][None, :, None]).sum(1)
            for s in range(t + 1):
                y = y + (torch.exp(F[t] - F[s]) * step[a + s] * (B[a + s] @ C[a + t]))[:, None] * x[a + s]
            got.append(y)
        S = torch.exp(F[-1])[:, None, None] * S
        for s in range(b - a):
            S = S + (torch.exp(F[-1] - F[s]) * step[a + s])[:, None, None] * B[a + s][None, :, None] * x[a + s][:, None, :]
    assert torch.allclose(torch.stack(got), torch.stack(want), rtol=1e-10, atol=1e-10)


def test_values_are_the_keys_behind_the_filter_and_before_the_rotation():
    """One head, one visible key at a time by a huge score: what comes out is the filtered key, unrotated, and the filter reaches
    back over the tokens before it."""
    m = left(1, 1, 2, 1.0, 3, None, {"dims": 2, "base": 10.0})
    W = {"q": torch.zeros(2, 2), "q.b": torch.zeros(2), "k": torch.eye(2), "k.b": torch.tensor([0.5, 0.0]), "q.conv": torch.ones(2, 3),
         "k.conv": torch.tensor([[1.0, 0.0, 2.0], [0.0, 1.0, 1.0]]), "sink": torch.tensor([-50.0]), "o": torch.eye(2)}
    W = {n: t.double() for n, t in W.items()}
    h = torch.tensor([[1.0, 1.0], [2.0, -1.0], [4.0, 3.0]]).double()
    out = P.attention(h, W, m)                                        # zero queries: equal weights over what is seen
    v = torch.tensor([[2 * 1.5, 1.0], [2 * 2.5, -1.0 + 1.0], [2 * 4.5 + 1.5, 3.0 - 1.0]]).double()
    assert torch.allclose(out, torch.stack([v[:t + 1].mean(0) for t in range(3)]), atol=1e-9)
    W["sink"] = torch.tensor([math.log(3.0)]).double()                # three keys of score 0 beside a sink of 3
    assert torch.allclose(P.attention(h, W, m)[2], v.sum(0) / 6, atol=1e-9)


def test_each_half_of_the_pair_is_divided_by_its_own_size():
    cfg = CONFIGS["X"]
    w = {n: t.double() for n, t in P.random_weights(cfg, 3).items()}
    W, m = P.sub(w, "l0.mix."), cfg["layers"][0]["mixer"]
    h = torch.randn(20, 72, generator=torch.Generator().manual_seed(0)).double()
    y = P.parallel_mixer(h, W, m, 1e-30)
    W2 = dict(W, **{"left.o": W["left.o"] * 7.0, "right.o": W["right.o"] * 0.01})
    assert torch.allclose(P.parallel_mixer(h, W2, m, 1e-30), y, rtol=1e-9, atol=1e-12)


def test_the_plain_model_is_causal_and_every_tensor_matters():
    w = P.random_weights(CFG, 1, dtype=torch.float32)
    toks = [3, 9, 1, 44, 20, 7, 7, 30, 12, 5, 100, 2, 2, 61, 17]
    a = P.forward(CFG, w, toks)
    b = P.forward(CFG, w, toks[:9] + [1, 2, 3, 4, 5, 6])
    assert torch.allclose(a[:9], b[:9], rtol=1e-9, atol=1e-9) and not torch.allclose(a[9:], b[9:], atol=1e-3)
    streams = []
    P.forward(CFG, w, toks, streams=streams)
    assert len(streams) == 7
    g = torch.Generator().manual_seed(5)
    for n in w:
        changed = P.forward(CFG, dict(w, **{n: w[n] + 0.3 * torch.randn(w[n].shape, generator=g)}), toks)
        assert float((changed - a).abs().max()) > 1e-3 * float(a.abs().max()), n
