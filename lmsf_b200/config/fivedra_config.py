"""The typed configuration of the Fivedra design, read from config.json.

config.json of this design is nested: `layers` lists every layer with its `type` (which mixer), the mixer's sizes (`mixer`) and
its feed-forward (`mlp`, or null for none); `embedding.scale`, `norm.eps`, `vocab` and `width` are global.  Every size and every
constant that may differ between models of the design is read from there (the number of distance buckets from the stored
table); nothing is assumed equal between layers.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Union

from .model_config import ConfigError

MIXER_TYPES = ("mingru", "parallel", "latent_attention")


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
class MinGRUMixer:
    width: int


@dataclass
class WindowAttention:
    """The left half of a `parallel` mixer: values are keys, a learned bias per distance bucket, a window."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    bias_max: float
    window: Optional[int] = None                          # mask.size; None: every earlier token is seen


@dataclass
class MatrixMemoryMixer:
    """The right half of a `parallel` mixer."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass
class ParallelMixer:
    left: WindowAttention
    right: MatrixMemoryMixer
    left_scale: float
    right_scale: float


@dataclass
class LatentMixer:
    heads: int
    dim: int                                             # unrotated query/key values per head
    vdim: int
    kv_rank: int
    q_rank: int
    rot_dim: int                                         # rotated query/key values per head
    rot_dims: int                                        # how many of those are rotated (the rest pass unchanged)
    rot_base: float
    scale: float
    scaling: Optional[Dict[str, float]] = None           # factor, original, fast, slow


@dataclass
class FivedraLayer:
    type: str
    mixer: Union[MinGRUMixer, ParallelMixer, LatentMixer]
    ff: Optional[int]                                    # hidden size of the feed-forward; None: the layer has none


def _parallel(m: Dict[str, Any], where: str) -> ParallelMixer:
    a, b = _need(m, "left", where), _need(m, "right", where)
    heads, dim = _pos_int(_need(a, "heads", where + ".left"), "left.heads"), _pos_int(_need(a, "dim", where + ".left"), "left.dim")
    kv_heads = _pos_int(a.get("kv_heads") or heads, "left.kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.left: {heads} heads over {kv_heads} kv heads")
    if a.get("vdim") not in (None, dim):
        raise ConfigError(f"config.json: {where}.left: values that are the keys have the keys' size {dim}, not {a['vdim']}")
    scale = _pos_number(a["scale"], "left.scale") if a.get("scale") is not None else dim ** -0.5
    left = WindowAttention(heads, kv_heads, dim, scale, _pos_number(_need(a, "bias_max", where + ".left"), "left.bias_max"))
    mask = a.get("mask")
    if mask and mask.get("size") is not None:
        left.window = _pos_int(mask["size"], "left.mask.size")
    right = MatrixMemoryMixer(_pos_int(_need(b, "heads", where + ".right"), "right.heads"),
                              _pos_int(_need(b, "dim", where + ".right"), "right.dim"),
                              _pos_int(_need(b, "vdim", where + ".right"), "right.vdim"),
                              _pos_number(_need(b, "gate_cap", where + ".right"), "right.gate_cap"))
    return ParallelMixer(left, right, _number(m.get("left_scale", 1.0), "left_scale"), _number(m.get("right_scale", 1.0), "right_scale"))


def _latent(m: Dict[str, Any], where: str) -> LatentMixer:
    get = lambda k: _pos_int(_need(m, k, where), k)
    rot = m.get("rot") or {}
    mixer = LatentMixer(get("heads"), get("dim"), get("vdim"), get("kv_rank"), get("q_rank"), get("rot_dim"), 0,
                        _pos_number(rot.get("base", 10000.0), "rot.base"), 0.0)
    mixer.rot_dims = _pos_int(rot.get("dims", mixer.rot_dim), "rot.dims")
    if mixer.rot_dims % 2 or mixer.rot_dims > mixer.rot_dim:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most rot_dim ({mixer.rot_dim})")
    mixer.scale = _pos_number(m["scale"], "scale") if m.get("scale") is not None else (mixer.dim + mixer.rot_dim) ** -0.5
    sc = rot.get("scaling")
    if sc:
        mixer.scaling = {k: _pos_number(_need(sc, k, where + ".rot.scaling"), f"rot.scaling.{k}") for k in ("factor", "original", "fast", "slow")}
        if mixer.rot_base <= 1:
            raise ConfigError(f"config.json: {where}.rot: stretched frequencies need a base above 1, got {mixer.rot_base}")
    return mixer


@dataclass
class FivedraConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: List[FivedraLayer]
    max_model_len: int = 1 << 20                         # bounded by the cache alone
    torch_dtype: str = "bfloat16"
    eos_token_ids: List[int] = field(default_factory=list)
    raw: Dict[str, Any] = field(default_factory=dict)

    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "FivedraConfig":
        vocab, width = _pos_int(_need(d, "vocab", "the model"), "vocab"), _pos_int(_need(d, "width", "the model"), "width")
        eps = _pos_number(_need(_need(d, "norm", "the model"), "eps", "norm"), "norm.eps")
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
            mixer = MinGRUMixer(_pos_int(_need(m, "width", at), "width")) if kind == "mingru" else \
                _parallel(m, at) if kind == "parallel" else _latent(m, at)
            f = L.get("mlp")
            ff = None
            if f:
                if f.get("kind", "dense") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {f['kind']!r} is not a feed-forward of this design (dense)")
                ff = _pos_int(_need(f, "ff", where + ".mlp"), "ff")
            layers.append(FivedraLayer(kind, mixer, ff))
        cfg = FivedraConfig(vocab, width, eps, scale, layers, raw=dict(d))
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
