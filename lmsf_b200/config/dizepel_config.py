"""The typed configuration of the Dizepel design, read from config.json.

config.json of this design is nested: `layers` lists every layer with its `type` (which mixer), the mixer's sizes (`mixer`, its two
halves under `left` and `right`) and its feed-forward (`mlp`, or null for none); `canon.taps`, `embedding.scale`, `loop`, `norm.eps`,
`vocab` and `width` are global.  Every size and every constant that may differ between models of the design is read from there;
nothing is assumed equal between layers.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .model_config import ConfigError

MIXER_TYPES = ("parallel",)


def _need(d: Dict[str, Any], key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: {where} lacks {key!r}")
    return d[key]


def _pos_int(v, what: str) -> int:
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"config.json: {what} must be a positive integer, got {v!r}")
    return v


def _number(v, what: str) -> float:
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {what} must be a number, got {v!r}")
    return float(v)


def _pos_number(v, what: str) -> float:
    x = _number(v, what)
    if not x > 0:
        raise ConfigError(f"config.json: {what} must be positive, got {v!r}")
    return x


@dataclass
class FilteredAttention:
    """The left half: queries and keys pass a short filter, values are the filtered keys before the rotation."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    conv: int                                            # taps of the filter on queries and keys
    softcap: Optional[float] = None
    rot_dims: int = 0
    rot_base: float = 10000.0
    scaling: Optional[Dict[str, float]] = None           # factor, original, fast, slow


@dataclass
class StateSpaceMixer:
    """The right half."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass
class ParallelMixer:
    left: FilteredAttention
    right: StateSpaceMixer


@dataclass
class DizepelLayer:
    mixer: ParallelMixer
    ff: Optional[int]                                    # hidden size of the feed-forward; None: the layer has none


def _left(a: Dict[str, Any], where: str) -> FilteredAttention:
    get = lambda k: _pos_int(_need(a, k, where), f"{where}.{k}")
    heads, dim = get("heads"), get("dim")
    kv_heads = _pos_int(a.get("kv_heads") or heads, where + ".kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: {heads} heads over {kv_heads} kv heads")
    if a.get("vdim") not in (None, dim):
        raise ConfigError(f"config.json: {where}: values that are the keys have the keys' size {dim}, not {a['vdim']}")
    scale = _pos_number(a["scale"], where + ".scale") if a.get("scale") is not None else dim ** -0.5
    m = FilteredAttention(heads, kv_heads, dim, scale, _pos_int(a.get("conv") or 1, where + ".conv"))
    if a.get("softcap"):
        m.softcap = _pos_number(a["softcap"], where + ".softcap")
    rot = a.get("rot")
    if rot:
        m.rot_dims = _pos_int(rot.get("dims", dim), where + ".rot.dims")
        m.rot_base = _pos_number(_need(rot, "base", where + ".rot"), where + ".rot.base")
        if m.rot_dims % 2 or m.rot_dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim ({dim}), got {m.rot_dims}")
        sc = rot.get("scaling")
        if sc:
            m.scaling = {k: _pos_number(_need(sc, k, where + ".rot.scaling"), f"{where}.rot.scaling.{k}") for k in ("factor", "original", "fast", "slow")}
            if m.rot_base <= 1:
                raise ConfigError(f"config.json: {where}.rot: stretched frequencies need a base above 1, got {m.rot_base}")
    return m


def _right(b: Dict[str, Any], where: str) -> StateSpaceMixer:
    get = lambda k: _pos_int(_need(b, k, where), f"{where}.{k}")
    m = StateSpaceMixer(get("heads"), get("vdim"), get("state"), _pos_int(b.get("groups") or 1, where + ".groups"),
                        _pos_int(b.get("conv") or 1, where + ".conv"), _pos_int(b.get("norm_groups") or 1, where + ".norm_groups"))
    if m.heads % m.groups:
        raise ConfigError(f"config.json: {where}: {m.heads} heads over {m.groups} groups")
    if (m.heads * m.vdim) % m.norm_groups:
        raise ConfigError(f"config.json: {where}.norm_groups: {m.norm_groups} parts of {m.heads * m.vdim} values")
    return m


@dataclass
class DizepelConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    canon_taps: int
    layers: List[DizepelLayer]
    has_loop: bool = False
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    max_model_len: int = 1 << 20                         # bounded by the cache alone
    torch_dtype: str = "bfloat16"
    eos_token_ids: List[int] = field(default_factory=list)
    raw: Dict[str, Any] = field(default_factory=dict)

    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "DizepelConfig":
        vocab, width = _pos_int(_need(d, "vocab", "the model"), "vocab"), _pos_int(_need(d, "width", "the model"), "width")
        eps = _pos_number(_need(_need(d, "norm", "the model"), "eps", "norm"), "norm.eps")
        taps = _pos_int(_need(_need(d, "canon", "the model"), "taps", "canon"), "canon.taps")
        scale = _number((d.get("embedding") or {}).get("scale", 1.0), "embedding.scale")
        raw_layers = _need(d, "layers", "the model")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = _need(L, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design ({', '.join(MIXER_TYPES)})")
            m, at = _need(L, "mixer", where), where + ".mixer"
            mixer = ParallelMixer(_left(_need(m, "left", at), at + ".left"), _right(_need(m, "right", at), at + ".right"))
            f, ff = L.get("mlp"), None
            if f:
                if f.get("kind", "dense") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {f['kind']!r} is not a feed-forward of this design (dense)")
                ff = _pos_int(_need(f, "ff", where + ".mlp"), where + ".mlp.ff")
            layers.append(DizepelLayer(mixer, ff))
        cfg = DizepelConfig(vocab, width, eps, scale, taps, layers, raw=dict(d))
        loop = d.get("loop")
        if loop:
            start, stop, times = int(_need(loop, "start", "loop")), int(_need(loop, "stop", "loop")), int(_need(loop, "times", "loop"))
            if not (0 <= start <= stop <= len(layers)) or times < 1:
                raise ConfigError(f"config.json: loop {loop!r} does not fit {len(layers)} layers")
            if stop > start:
                cfg.loop_start, cfg.loop_stop, cfg.loop_times, cfg.has_loop = start, stop, times, True
        if d.get("max_len"):
            cfg.max_model_len = _pos_int(d["max_len"], "max_len")
        dt = d.get("torch_dtype", d.get("dtype"))
        if dt is not None:
            cfg.torch_dtype = str(dt).replace("torch.", "")
        eos = d.get("eos_token_id")
        if eos is not None:
            cfg.eos_token_ids = [int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos])]
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)
