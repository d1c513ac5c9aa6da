"""Dizepel: the description of the decoder as data, and its registry entry.

A scaled embedding; layers with a layer norm before and after each branch, whose mixer and feed-forward read the first norm's
output plus a short causal filter of it over time; one mixer, a parallel pair: attention whose queries and keys pass a short
filter, whose values are the filtered keys before a partial rotation with stretched frequencies, with capped scores and a learned
sink per head, beside a selective state space; each half is normed by its root mean square and half the sum goes on; a
feed-forward with a polynomial activation whose powers are normed, or none; a span of layers that runs several times with the same
weights, a vector added to the stream at the start of each pass; a final layer norm and a head.  Tensor names: `embed`,
`loop.step`, `final.norm`, `head`, and `l<i>.` + `norm1`, `norm1b`, `norm2`, `norm2b`, `canon1`, `canon2`, `mix.left.*`,
`mix.right.*`, `mlp.*`.
"""
from __future__ import annotations

from ..config.dizepel_config import DizepelConfig, ParallelMixer
from ..config.registry import register_architecture
from ..parts.base import LayerCall, LayerSpec, ModelSpec, PartSpec


def _parallel(D: int, eps: float, m: ParallelMixer, x: str) -> PartSpec:
    a, b, l, r = m.left, m.right, x + "left.", x + "right."
    rope = None
    if a.rot_dims:
        sc = a.scaling
        rope = PartSpec("rotary", dict(rot_dim=a.rot_dims, theta=a.rot_base, is_neox=True,
                                       **(dict(scaling_type="yarn", factor=sc["factor"], original_max_position_embeddings=sc["original"],
                                               beta_fast=sc["fast"], beta_slow=sc["slow"]) if sc else {})))
    left = PartSpec("paged_attention",
                    dict(hidden_size=D, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, position_encoding=rope,
                         scale=a.scale, softcap=a.softcap, bias=True, out_bias=False, values_are_keys=True, qk_filter=a.conv,
                         learned_sink=True),
                    {"qkv": [l + "q", l + "k"], "qkv_bias": [l + "q.b", l + "k.b"], "qk_filter": [l + "q.conv", l + "k.conv"],
                     "sink": l + "sink", "o": l + "o"})
    right = PartSpec("selective_state_space",
                     dict(hidden_size=D, num_heads=b.heads, head_dim=b.vdim, state_size=b.state, groups=b.groups, conv_taps=b.conv,
                          norm_groups=b.norm_groups, eps=eps),
                     {"in_proj": r + "in", "conv": r + "conv", "conv_bias": r + "conv.b", "dt_bias": r + "dt_bias", "a_log": r + "A_log",
                      "skip": r + "D", "norm": r + "norm", "o": r + "o"})
    return PartSpec("normed_parallel_mixers", dict(mixer_left=left, mixer_right=right, eps=eps, factor=0.5),
                    {"left_norm": l + "out", "right_norm": r + "out"})


def dizepel_spec(cfg: DizepelConfig) -> ModelSpec:
    D = cfg.width
    norm = lambda name: PartSpec("layernorm", dict(hidden_size=D, eps=cfg.eps), {"weight": name})
    filt = lambda name: PartSpec("filter_shift", dict(hidden_size=D, taps=cfg.canon_taps), {"filter": name})
    layers, ignored = [], []
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer_norm": norm(p + "norm1"), "mixer_shift": filt(p + "canon1"), "mixer": _parallel(D, cfg.eps, L.mixer, p + "mix."),
                 "mixer_post_norm": norm(p + "norm1b")}
        if L.ff is None:
            ignored += [rf"^l{i}\.{n}$" for n in ("norm2", "norm2b", "canon2")]
        else:
            parts.update(ffn_norm=norm(p + "norm2"), ffn_shift=filt(p + "canon2"), ffn_post_norm=norm(p + "norm2b"),
                         feed_forward=PartSpec("plain_mlp", dict(hidden_size=D, intermediate_size=L.ff, eps=cfg.eps, activation="poly_norm"),
                                               {"up": p + "mlp.up", "down": p + "mlp.down", "act": p + "mlp.act"}))
        layers.append(LayerSpec("sandwich_norm", parts))
    entries, order = [], [LayerCall(i) for i in range(len(layers))]
    if cfg.has_loop:
        entries.append(PartSpec("loop_entry", dict(hidden_size=D, times=cfg.loop_times, readd_first=False, step_vector=True),
                                {"step": "loop.step"}))
        passes = [LayerCall(i, entry=0, entry_pass=t) if i == cfg.loop_start else LayerCall(i)
                  for t in range(cfg.loop_times) for i in range(cfg.loop_start, cfg.loop_stop)]
        order = order[:cfg.loop_start] + passes + order[cfg.loop_stop:]
    else:
        ignored.append(r"^loop\.step$")
    return ModelSpec(
        hidden_size=D, vocab_size=cfg.vocab, max_model_len=cfg.max_model_len,
        embedding=PartSpec("token_embedding", dict(vocab_size=cfg.vocab, hidden_size=D, scale=cfg.embed_scale, as_stream=True),
                           {"weight": "embed"}),
        layers=layers, order=order, entries=entries,
        final_norm=norm("final.norm"),
        lm_head=PartSpec("dense", dict(in_features=D, out_features=cfg.vocab, out_dtype="float32"), {"weight": "head"}),
        eos_token_ids=list(cfg.eos_token_ids), ignored_weights=ignored,
    )


register_architecture("Dizepel", DizepelConfig.from_dict, dizepel_spec, aliases=("dizepel",))
