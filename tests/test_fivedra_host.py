"""Host side of the Fivedra design: its configuration, its description as data, its tensor names, the tables made on the host,
and the identities that the engine's kernels rest on, checked on the plain implementation alone."""
import copy
import json
import math

import pytest
import torch

import plain_fivedra as P
from fivedra_configs import CONFIGS

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
    assert [L.type for L in typed.layers] == ["parallel", "mingru", "latent_attention", "parallel"] and typed.embed_scale == 3.0
    groups, _ = plan_groups(model)
    # one plane everywhere: keys that are values (heads padded to multiples of 16), and rank + rotated part in one row
    by_calls = {tuple(g.calls): (g.spec.num_kv_heads, g.spec.head_dim, g.spec.planes, g.spec.window) for g in groups}
    assert by_calls == {(0,): (2, 32, 1, 21), (2,): (1, 64, 1, None), (3,): (2, 16, 1, 50)}
    # a parallel layer has pages AND a state slot: S, then n and m once per 64 value columns
    assert [model.call_state_spec(j).shape[0] if model.call_state_spec(j) else None for j in range(4)] == \
        [3 * 10 * 18 + 3 * 10 + 3, 50, None, 33 * 70 + 2 * 33 + 2]
    assert model.blocks[2].feed_forward is None and model.blocks[2].ffn_norm is None
    assert [b.mixer.out_scale for b in model.blocks] == [0.7, 1.0, 1.0, -0.4]
    assert all(getattr(p, "graph_safe", False) for p, _ in model.parts_with_specs())


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


def test_the_number_of_buckets_is_the_stored_tables():
    from lmsf_b200.parts.rope import BucketedDistanceBias
    part = BucketedDistanceBias(num_heads=3, far=40)
    spec = part.weight_specs()["table"]
    assert spec.matches(0, (7, 3)) and spec.matches(0, (32, 3)) and not spec.matches(0, (7, 2)) and not spec.matches(0, (7,))
    for B in (1, 2, 7, 32):
        part.set_weights({"table": torch.arange(3.0 * B).view(B, 3)})
        part.prepare(torch.float32, torch.device("cpu"))
        t = part.score_distance_table()
        assert part.buckets == B and t.shape[0] == 3
        for n in range(100):
            want = P.bucket(n, B, 40) if B > 1 else 0
            assert t[:, min(n, t.shape[1] - 1)].tolist() == part.table[want].tolist(), (B, n)


@pytest.mark.parametrize("count,far", [(16, 128), (32, 128), (8, 20), (10, 1000), (7, 13), (16, 9), (16, 8), (64, 33)])
def test_buckets_are_single_distances_first_and_then_widen(count, far):
    from lmsf_b200.parts.rope import distance_bucket
    half = count // 2
    got = [distance_bucket(n, count, far) for n in range(3 * far + 40)]
    assert got[:half] == list(range(half)) and all(b - a in range(0, count) for a, b in zip(got, got[1:]))      # never falls
    assert all(b == count - 1 for b in got[max(far, half):])
    if far > half:
        assert got == [P.bucket(n, count, far) for n in range(len(got))]


def test_stretched_frequencies_are_the_plain_ones():
    from lmsf_b200.parts.rope import rope_inverse_frequencies, yarn_magnitude
    for rot in (dict(dims=12, base=500.0, scaling=dict(factor=4.0, original=40, fast=4.0, slow=0.5)),
                dict(dims=64, base=1.0e4, scaling=dict(factor=32.0, original=4096, fast=32.0, slow=1.0)),
                dict(dims=2, base=50.0, scaling=dict(factor=2.0, original=64, fast=8.0, slow=4.0)),
                dict(dims=16, base=1.0e6, scaling=dict(factor=1.0, original=1024, fast=1.0, slow=1.0))):
        sc = rot["scaling"]
        want, mult = P.rotary_frequencies(rot)
        got = rope_inverse_frequencies(rot["dims"], rot["base"], "yarn", factor=sc["factor"],
                                       original_max_position_embeddings=sc["original"], beta_fast=sc["fast"], beta_slow=sc["slow"])
        assert got == pytest.approx(want, rel=1e-12) and yarn_magnitude(sc["factor"]) == pytest.approx(mult, rel=1e-12)
    # fast pairs keep their frequency, slow ones are divided by the factor
    f, _ = P.rotary_frequencies(dict(dims=64, base=1.0e4, scaling=dict(factor=32.0, original=4096, fast=32.0, slow=1.0)))
    assert f[0] == 1.0 and f[-1] == pytest.approx(1.0e4 ** (-62 / 64) / 32.0)


@pytest.mark.parametrize("change,needle", [
    (lambda c: c["layers"][0].update(type="convolution"), "type"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("bias_max"), "bias_max"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(vdim=48), "values that are the keys"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"].update(width=-1), "width"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
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
    del w["l2.mix.sink"]
    w["l0.mix.left.rel"] = torch.ones(16, 3, dtype=torch.bfloat16)
    w["l9.extra"] = torch.ones(2, dtype=torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    write_safetensors(str(tmp_path / "model.safetensors"), [(n, t.dtype, tuple(t.shape)) for n, t in w.items()], lambda n: w[n])
    with pytest.raises(WeightError) as e:
        check_tensors(model, open_model_tensors(str(tmp_path)), str(tmp_path))
    assert e.value.missing == ["l2.mix.sink"] and e.value.unexpected == ["l9.extra"] and e.value.wrong_shape[0][0] == "l0.mix.left.rel"


def test_a_block_that_does_not_multiply_its_mixer_refuses_one_that_asks_for_it():
    from lmsf_b200.parts.base import LayerSpec
    from lmsf_b200.parts.decoder import DecoderModel
    typed, model = build(CFG)
    spec = copy.copy(model.spec)
    spec.layers = [LayerSpec("pre_norm", model.spec.layers[0].parts)] + list(model.spec.layers[1:])
    with pytest.raises(ValueError, match="factor"):
        DecoderModel(spec)


def test_norm_weights_around_zero_keep_their_digits():
    """1 + w has more digits than a stored bfloat16: the sum stays in float32."""
    from lmsf_b200.parts.norm import RMSNorm
    n = RMSNorm(hidden_size=3, eps=1e-5, weight_offset=1.0)
    w = torch.tensor([0.0013, -0.4, 0.25], dtype=torch.bfloat16)
    n.set_weights({"weight": w})
    assert n.weight.dtype == torch.float32 and torch.equal(n.weight, 1.0 + w.float())


# ----------------------------------------------------------------------------- identities

def test_chunks_of_the_matrix_memory_with_a_maximum_of_their_own_equal_the_recurrence():
    """S, n and m after a chunk from what the chunk adds (scaled by its own maximum) and what it found; outputs from the state
    before the chunk and the gated score matrix: the algebra of the three kernels for long portions."""
    g = torch.Generator().manual_seed(0)
    m = dict(heads=1, dim=5, vdim=4, gate_cap=6.0)
    T, D, C = 37, 9, 8
    W = {n: torch.randn(*s, generator=g).double() for n, s in dict(q=(5, D), k=(5, D), v=(4, D), g=(4, D), o=(4, 4), i=(1, D), f=(1, D)).items()}
    W.update({"i.b": torch.tensor([0.5]).double(), "f.b": torch.tensor([1.5]).double(), "norm": torch.ones(4).double(), "o": torch.eye(4).double()})
    h = torch.randn(T, D, generator=g).double() * 2
    want = P.matrix_memory(h, W, m, 1e-9)
    cap = m["gate_cap"]
    li, lf = cap * torch.tanh((h @ W["i"].T + 0.5) / cap)[:, 0], P.log_sigmoid(cap * torch.tanh((h @ W["f"].T + 1.5) / cap))[:, 0]
    q, k, v = h @ W["q"].T * 5 ** -0.5, h @ W["k"].T, h @ W["v"].T
    S, n, top = torch.zeros(5, 4).double(), torch.zeros(5).double(), 0.0
    rows = []
    for a in range(0, T, C):
        b = min(a + C, T)
        F = torch.cumsum(lf[a:b], 0)
        e = F[:, None] - F[None, :] + li[None, a:b]
        e = e.masked_fill(torch.ones_like(e).triu(1).bool(), -math.inf)
        r = e.max(1).values
        Pm = torch.exp(e - r[:, None]) * (q[a:b] @ k[a:b].T)
        mt = torch.maximum(F + top, r)
        inter, intra = torch.exp(F + top - mt), torch.exp(r - mt)
        o = inter[:, None] * (q[a:b] @ S) + intra[:, None] * (Pm @ v[a:b])
        nq = inter * (q[a:b] @ n) + intra * Pm.sum(1)
        rows.append(o / (torch.maximum(nq.abs(), torch.exp(-mt)) + 1e-6)[:, None])
        we = F[-1] - F + li[a:b]
        c = we.max()
        w = torch.exp(we - c)[:, None] * k[a:b]
        new = max(float(F[-1]) + top, float(c))
        S = math.exp(float(F[-1]) + top - new) * S + math.exp(float(c) - new) * (w.T @ v[a:b])
        n = math.exp(float(F[-1]) + top - new) * n + math.exp(float(c) - new) * w.sum(0)
        top = new
    y = P.rms(torch.cat(rows), 1e-9) * P.sigmoid(h @ W["g"].T)
    assert torch.allclose(y, want, rtol=1e-8, atol=1e-9)


def test_the_running_maximum_starts_at_zero_and_the_floor_counts():
    """With all gates closed the denominator is the floor, not n . q: a maximum that started at minus infinity would give the
    value itself, whatever the gate."""
    m = dict(heads=1, dim=1, vdim=2, gate_cap=50.0)
    one = torch.ones(1, 1).double()
    W = {"q": one, "k": one, "v": torch.tensor([[2.0], [3.0]]).double(), "g": torch.zeros(2, 1).double(), "o": torch.eye(2).double(),
         "i": 0 * one, "f": 0 * one, "i.b": torch.tensor([-4.0]).double(), "f.b": torch.tensor([0.0]).double(), "norm": torch.ones(2).double()}
    eps = 1.0                                                        # a large eps, so that the head's norm keeps the size
    got = P.matrix_memory(torch.ones(1, 1).double(), W, m, eps)[0]
    cap = 50.0
    i, f = cap * math.tanh(-4.0 / cap), math.log(0.5)
    mt = max(f, i)
    o = math.exp(i - mt) * torch.tensor([2.0, 3.0]).double() / (max(math.exp(i - mt), math.exp(-mt)) + 1e-6)
    assert torch.allclose(got, 0.5 * P.rms(o, eps), rtol=1e-9)
    assert float(o.max()) < 0.1


def test_steps_of_the_min_gru_compose():
    """S -> a S + b: two steps are (a2 a1, a2 b1 + b2), so lanes of tokens may be scanned in parallel; 1 - z is sigmoid(-logit)."""
    g = torch.Generator().manual_seed(1)
    z, u = torch.randn(9, generator=g).double(), torch.randn(9, generator=g).double()
    a, b = P.sigmoid(-z), P.sigmoid(z) * torch.where(u >= 0, u + 0.5, P.sigmoid(u))
    S = 0.7
    for x, y in zip(a, b):
        S = float(x) * S + float(y)
    A, B = 1.0, 0.0
    for x, y in zip(a, b):
        A, B = float(x) * A, float(x) * B + float(y)
    assert abs(A * 0.7 + B - S) < 1e-12
    W = {"z": torch.zeros(1, 1), "x": torch.ones(1, 1), "g": torch.ones(1, 1), "o": torch.ones(1, 1), "z.b": torch.tensor([40.0]), "x.b": torch.zeros(1)}
    W = {n: t.double() for n, t in W.items()}
    y = P.min_gru_mixer(torch.tensor([[2.0], [-3.0]]).double(), W)[:, 0]      # z = 1: the state is the candidate
    want = [2.5 * 2.0 / (1 + math.exp(-2.0)), 1 / (1 + math.exp(3.0)) * -3.0 / (1 + math.exp(3.0))]
    assert y.tolist() == pytest.approx(want, rel=1e-9)


def test_one_in_the_denominator_and_a_window_whose_edge_counts():
    m = dict(heads=1, kv_heads=1, dim=2, scale=1.0, bias_max=8, mask={"size": 3})
    W = {"q": torch.zeros(2, 2), "q.b": torch.zeros(2), "k": torch.eye(2), "k.b": torch.tensor([0.0, 1.0]), "rel": torch.zeros(4, 1), "o": torch.eye(2)}
    W = {n: t.double() for n, t in W.items()}
    h = torch.zeros(6, 2).double()
    h[:, 0] = torch.arange(6.0)
    out = P.window_attention(h, W, m)
    assert out[0].tolist() == pytest.approx([0.0, 0.5])               # one key of score 0 beside the one: half its value
    assert out[5].tolist() == pytest.approx([(3 + 4 + 5) / 4, 0.75])  # keys 3, 4, 5 and the one; the value carries the key's bias
    W["rel"] = torch.tensor([[0.0], [0.0], [5.0], [0.0]]).double()    # bucket 2: distances 2 and 3 of 8
    assert P.bucket(2, 4, 8) == 2 and P.bucket(3, 4, 8) == 2 and P.bucket(4, 4, 8) == 3
    assert float(P.window_attention(h, W, m)[5, 0]) < 3.1             # the key at distance 2 takes nearly all


def test_the_plain_model_is_causal():
    w = P.random_weights(CFG, 1, dtype=torch.float32)
    toks = [3, 9, 1, 44, 20, 7, 7, 30, 12, 5, 100, 2, 2, 61, 17]
    a = P.forward(CFG, w, toks)
    b = P.forward(CFG, w, toks[:9] + [1, 2, 3, 4, 5, 6])
    assert torch.allclose(a[:9], b[:9], rtol=1e-9, atol=1e-9) and not torch.allclose(a[9:], b[9:], atol=1e-3)
    streams = []
    P.forward(CFG, w, toks, streams=streams)
    assert len(streams) == 4
