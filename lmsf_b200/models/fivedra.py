"""Fivedra: the description of the decoder as data, and its registry entry.

A scaled embedding; layers whose two branches run side by side behind a norm each, x <- x + (mixer(norm1(x)) + ff(norm2(x))),
the norms' weights stored around zero; three mixers: a minGRU (an element-wise gated recurrence), a parallel pair (attention
whose values are its keys, with a learned bias per distance bucket, a sliding window and one more in the softmax's denominator;
beside it the matrix memory of xLSTM), and attention over a cached low-rank vector plus one rotated key part shared by all
heads, with low-rank queries, stretched frequencies and a learned sink per head; a feed-forward with the square of relu, or
none; a final norm and a head.  Tensor names: `embed`, `final.norm`, `head`, and `l<i>.` + `norm1`, `norm2`, `mix.*`, `mlp.*`.
"""
from __future__ import annotations

from ..config.fivedra_config import FivedraConfig, LatentMixer, MinGRUMixer, ParallelMixer
from ..config.registry import register_architecture
from ..parts.base import LayerCall, LayerSpec, ModelSpec, PartSpec


def _min_gru(D: int, m: MinGRUMixer, x: str) -> PartSpec:
    return PartSpec("min_gru", dict(hidden_size=D, width=m.width),
                    {"zxg": [x + "z", x + "x", x + "g"], "z_bias": x + "z.b", "x_bias": x + "x.b", "o": x + "o"})


def _parallel(D: int, eps: float, m: ParallelMixer, x: str) -> PartSpec:
    a, b, l, r = m.left, m.right, x + "left.", x + "right."
    bias = PartSpec("bucketed_distance_bias", dict(num_heads=a.heads, far=a.bias_max), {"table": l + "rel"})
    left = PartSpec("paged_attention",
                    dict(hidden_size=D, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, position_encoding=bias,
                         window=a.window, scale=a.scale, bias=True, out_bias=False, values_are_keys=True, unit_sink=True),
                    {"qkv": [l + "q", l + "k"], "qkv_bias": [l + "q.b", l + "k.b"], "o": l + "o"})
    right = PartSpec("matrix_memory",
                     dict(hidden_size=D, num_heads=b.heads, head_dim=b.dim, value_dim=b.vdim, gate_cap=b.gate_cap, eps=eps),
                     {"in_proj": [r + n for n in ("q", "k", "v", "g", "i", "f")], "i_bias": r + "i.b", "f_bias": r + "f.b",
                      "norm": r + "norm", "o": r + "o"})
    return PartSpec("parallel_mixers", dict(mixer_left=left, mixer_right=right, left_scale=m.left_scale, right_scale=m.right_scale))


def _latent(D: int, eps: float, m: LatentMixer, x: str) -> PartSpec:
    return PartSpec("latent_attention",
                    dict(hidden_size=D, num_heads=m.heads, head_dim=m.dim, value_dim=m.vdim, kv_rank=m.kv_rank, eps=eps,
                         scale=m.scale, window=None, gate=False, rope_dim=m.rot_dim, rope_dims=m.rot_dims, rope_base=m.rot_base,
                         rope_interleaved=True, rope_scaling=m.scaling, sink=True, q_rank=m.q_rank),
                    {"qcg": [x + "dq", x + "dkv"], "q_norm": x + "dq.norm", "uq": x + "uq", "c_norm": x + "dkv.norm",
                     "uk": x + "uk", "uv": x + "uv", "o": x + "o", "sink": x + "sink"})


def fivedra_spec(cfg: FivedraConfig) -> ModelSpec:
    D = cfg.width
    norm = lambda name: PartSpec("rmsnorm", dict(hidden_size=D, eps=cfg.eps, weight_offset=1.0), {"weight": name})
    layers, ignored = [], []
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}.", L.mixer
        x = p + "mix."
        mixer = _min_gru(D, m, x) if L.type == "mingru" else \
            _parallel(D, cfg.eps, m, x) if L.type == "parallel" else _latent(D, cfg.eps, m, x)
        parts = {"mixer_norm": norm(p + "norm1"), "mixer": mixer}
        if L.ff is None:
            ignored.append(rf"^l{i}\.norm2$")
        else:
            parts.update(ffn_norm=norm(p + "norm2"),
                         feed_forward=PartSpec("plain_mlp", dict(hidden_size=D, intermediate_size=L.ff, activation="relu2"),
                                               {"up": p + "mlp.up", "down": p + "mlp.down"}))
        layers.append(LayerSpec("parallel_norms", parts))
    return ModelSpec(
        hidden_size=D, vocab_size=cfg.vocab, max_model_len=cfg.max_model_len,
        embedding=PartSpec("token_embedding", dict(vocab_size=cfg.vocab, hidden_size=D, scale=cfg.embed_scale, as_stream=True),
                           {"weight": "embed"}),
        layers=layers, order=[LayerCall(i) for i in range(len(layers))],
        final_norm=norm("final.norm"),
        lm_head=PartSpec("dense", dict(in_features=D, out_features=cfg.vocab, out_dtype="float32"), {"weight": "head"}),
        eos_token_ids=list(cfg.eos_token_ids), ignored_weights=ignored,
    )


register_architecture("Fivedra", FivedraConfig.from_dict, fivedra_spec, aliases=("fivedra",))
