"""Rotary position encoding.

The reference builds a cos/sin table once per process with base 10000 whatever config.json says
(core/src/model_executor/layers/rotary_embedding.rs:8-29, :104-110; vllm/src/pos_encoding.rs:8-36)
and rotates NeoX-style in the model dtype (vllm/kernels/pos_encoding_kernels.cu:12-77).  Here the
base, the rotated width, the pairing and the frequency scaling are parameters; frequencies are
computed in float64 on the host and stored as float32, angles are position * inv_freq in float32
inside the kernel, so there is no table and no cap on positions.
"""
from __future__ import annotations

import math
from typing import List, Optional, Tuple

import torch

from .. import kernels
from .base import ANY_SIZE, PositionEncoding, StepContext, WeightSpec, register_part


def rope_inverse_frequencies(rot_dim: int, theta: float, scaling_type: str = "default", factor: float = 1.0,
                             low_freq_factor: float = 1.0, high_freq_factor: float = 4.0,
                             original_max_position_embeddings: float = 8192, beta_fast: float = 32.0,
                             beta_slow: float = 1.0) -> List[float]:
    """f_i = theta^(-2i/rot_dim), then by scaling type:
    linear: f_i / factor.
    llama3: wavelength 2 pi / f_i shorter than L0/high keeps f_i, longer than L0/low gives f_i / factor,
            between them an interpolation with s = (L0 / wavelength - low) / (high - low).
    yarn: pairs that turn more than beta_fast times within L0 positions keep f_i, pairs that turn less than beta_slow times
            get f_i / factor, between them (counted in pairs) a linear ramp; `yarn_magnitude` goes with it."""
    inv = [theta ** (-(2.0 * i) / rot_dim) for i in range(rot_dim // 2)]
    if scaling_type == "default":
        return inv
    if scaling_type == "linear":
        return [f / factor for f in inv]
    if scaling_type == "llama3":
        out = []
        l0 = float(original_max_position_embeddings)
        for f in inv:
            wavelen = 2.0 * math.pi / f
            if wavelen < l0 / high_freq_factor:
                out.append(f)
            elif wavelen > l0 / low_freq_factor:
                out.append(f / factor)
            else:
                s = (l0 / wavelen - low_freq_factor) / (high_freq_factor - low_freq_factor)
                out.append((1.0 - s) * f / factor + s * f)
        return out
    if scaling_type == "yarn":
        pair_of = lambda turns: rot_dim * math.log(original_max_position_embeddings / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
        lo = max(math.floor(pair_of(beta_fast)), 0)
        hi = min(math.ceil(pair_of(beta_slow)), rot_dim - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(rot_dim // 2)]
        return [f / factor * r + f * (1.0 - r) for f, r in zip(inv, ramp)]
    raise ValueError(f"unknown rope scaling type {scaling_type!r}")


def yarn_magnitude(factor: float) -> float:
    """What cos and sin are multiplied by where positions are stretched by `factor` the yarn way."""
    return 0.1 * math.log(factor) + 1.0


@register_part("position_encoding", "rotary")
class RotaryEmbedding(PositionEncoding):
    graph_safe = True

    def __init__(self, rot_dim: int, theta: float = 10000.0, is_neox: bool = True, scaling_type: str = "default",
                 factor: float = 1.0, low_freq_factor: float = 1.0, high_freq_factor: float = 4.0,
                 original_max_position_embeddings: float = 8192, beta_fast: float = 32.0, beta_slow: float = 1.0):
        if rot_dim <= 0 or rot_dim % 2:
            raise ValueError(f"rotary width must be a positive even number, got {rot_dim}")
        self.rot_dim = int(rot_dim)
        self.is_neox = bool(is_neox)
        self.inv_freq_host = rope_inverse_frequencies(rot_dim, float(theta), scaling_type, float(factor),
                                                      float(low_freq_factor), float(high_freq_factor),
                                                      original_max_position_embeddings, float(beta_fast), float(beta_slow))
        # what cos and sin are multiplied by (only parts that say so take a rotation that also stretches)
        self.mult = yarn_magnitude(float(factor)) if scaling_type == "yarn" else 1.0
        self.inv_freq: Optional[torch.Tensor] = None

    def prepare(self, dtype: torch.dtype, device: torch.device) -> None:
        self.inv_freq = torch.tensor(self.inv_freq_host, dtype=torch.float64).to(torch.float32).to(device)

    def fused_rotary(self) -> Optional[Tuple[torch.Tensor, int, bool]]:
        return self.inv_freq, self.rot_dim, self.is_neox

    def rotary_multiplier(self) -> float:
        return self.mult

    def apply(self, ctx: StepContext, q, k, n_q_heads, n_kv_heads, head_dim) -> None:
        kernels.rope_cache_write(q, None, None, ctx.positions, None, None, 0, None, self.inv_freq, self.rot_dim,
                                 self.is_neox, n_q_heads, 0, head_dim)
        if k is not None:
            kernels.rope_cache_write(k, None, None, ctx.positions, None, None, 0, None, self.inv_freq, self.rot_dim,
                                     self.is_neox, n_kv_heads, 0, head_dim)


@register_part("position_encoding", "none")
class NoPositionEncoding(PositionEncoding):
    graph_safe = True

    def __init__(self):
        pass

    def apply(self, ctx, q, k, n_q_heads, n_kv_heads, head_dim) -> None:
        return None


@register_part("position_encoding", "distance_bias")
class DistanceBias(PositionEncoding):
    """Positions enter the scores, not q and k: slope[head] * (key position - query position) is added to every scaled
    score (the reference's decode kernel takes such slopes, vllm/kernels/attention/attention_kernels.cu:144-145,
    :232-234, through layers/attention.rs:58-83; no model of its Llama path sets them).  The slopes are parameters, one
    per query head.  Only the generic attention kernel takes them, so an attention part with this encoding runs on that
    kernel in bfloat16 too: right, and slow."""
    graph_safe = True

    def __init__(self, slopes):
        self.slopes_host = [float(v) for v in slopes]
        if not self.slopes_host:
            raise ValueError("a distance bias needs one slope per query head")
        self.slopes: Optional[torch.Tensor] = None

    def prepare(self, dtype, device) -> None:
        self.slopes = torch.tensor(self.slopes_host, dtype=torch.float32, device=device)

    def apply(self, ctx, q, k, n_q_heads, n_kv_heads, head_dim) -> None:
        return None

    def score_slopes(self) -> Optional[torch.Tensor]:
        return self.slopes


@register_part("position_encoding", "log_distance_bias")
class LogDistanceBias(PositionEncoding):
    """Positions enter the scores, not q and k: r1[head] * log(1 + r2[head] * (query position - key position)) is taken
    off every scaled score.  r1 and r2 are learned, one number each per query head (weights `r1`, `r2`)."""
    graph_safe = True

    def __init__(self, num_heads: int):
        self.num_heads = int(num_heads)
        self.r1: Optional[torch.Tensor] = None
        self.r2: Optional[torch.Tensor] = None
        self._r: Optional[Tuple[torch.Tensor, torch.Tensor]] = None

    def weight_specs(self):
        return {"r1": WeightSpec([(self.num_heads,)], keep_fp32=True), "r2": WeightSpec([(self.num_heads,)], keep_fp32=True)}

    def prepare(self, dtype, device) -> None:
        self._r = (self.r1.float().contiguous(), self.r2.float().contiguous())

    def apply(self, ctx, q, k, n_q_heads, n_kv_heads, head_dim) -> None:
        return None

    def score_log_bias(self) -> Optional[Tuple[torch.Tensor, torch.Tensor]]:
        return self._r


def distance_bucket(n: int, count: int, far: float) -> int:
    """Which of `count` learned entries serves the distance n >= 0: the first half serve one distance each, the others ranges
    that widen with the logarithm of the distance, the last one everything from `far` on."""
    half = count // 2
    if n < half:
        return n
    if half == 0 or far <= half:
        return count - 1
    return min(count - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (count - half)))


@register_part("position_encoding", "bucketed_distance_bias")
class BucketedDistanceBias(PositionEncoding):
    """Positions enter the scores, not q and k: a learned number per (bucket of the distance, query head) is added to every
    scaled score (weight `table` [buckets, heads]; see `distance_bucket`).  The attention kernels take it spread out over the
    distances 0 .. far, float32 [heads, entries], whose last entry serves every larger distance.  `buckets` None: as many as
    the stored table has rows."""
    graph_safe = True

    def __init__(self, num_heads: int, far: float, buckets: Optional[int] = None):
        self.num_heads, self.far = int(num_heads), float(far)
        self.buckets = int(buckets) if buckets is not None else None
        if (self.buckets is not None and self.buckets < 1) or not self.far > 0:
            raise ValueError(f"a distance bias of {buckets} buckets up to distance {far}")
        self.table: Optional[torch.Tensor] = None
        self._spread: Optional[torch.Tensor] = None

    def weight_specs(self):
        return {"table": WeightSpec([(self.buckets if self.buckets is not None else ANY_SIZE, self.num_heads)], keep_fp32=True)}

    def set_weights(self, tensors) -> None:
        super().set_weights(tensors)
        if "table" in tensors:
            self.buckets = int(self.table.shape[0])

    def bucket_list(self) -> List[int]:
        """The bucket of every distance up to the first that, with all larger ones, belongs to the last bucket."""
        out = [distance_bucket(0, self.buckets, self.far)]
        while out[-1] < self.buckets - 1:
            out.append(distance_bucket(len(out), self.buckets, self.far))
        return out

    def prepare(self, dtype, device) -> None:
        which = torch.tensor(self.bucket_list(), dtype=torch.long, device=self.table.device)
        self._spread = self.table.float()[which].t().contiguous().to(device)

    def apply(self, ctx, q, k, n_q_heads, n_kv_heads, head_dim) -> None:
        return None

    def score_distance_table(self) -> Optional[torch.Tensor]:
        return self._spread
