"""Two mixers side by side that read the same input.

`parallel_mixers`: their outputs are added with a factor each,

  out = left_scale * attention(h) + right_scale * memory(h)

The left one is attention whose values are its keys, the right one a matrix memory.  Their matrices are merged when the weights
are on the device: one product for everything that reads h (queries, keys, and the memory's q, k, v, gates), one for both
output projections ([left | right] side by side).  The right factor is applied to the memory's float32 output before it is
rounded; the left one is asked of the block (`Mixer.out_scale`), which adds the result to the float32 stream: nothing is
rounded on its account.  The pages of the cache are the left mixer's, the state slot the right one's.

`normed_parallel_mixers`: each output is divided by its root mean square over the width and multiplied by a weight of its own,

  out = factor * (left / rms(left) * w_left + right / rms(right) * w_right)

The left one is attention whose queries and keys pass a filter, the right one a selective state space.  What reads h is one product
again; the two output products stay apart, and the block's kernel joins them (`BranchPair`): nothing is rounded between the two
norms and the sum into the stream.  A state slot holds the right mixer's state and behind it the left one's carried inputs.
"""
from __future__ import annotations

import os
from typing import Dict, Optional

import torch

from .base import BranchPair, KVCacheSpec, LayerCache, Mixer, StateSpec, StepContext, WeightSpec, register_part
from .linear import matmul_tn


CONCURRENT = os.environ.get("LMSF_CONCURRENT_MIXERS", "1") != "0"    # steps of single tokens: the two halves on two streams
_SIDE_STREAMS: Dict[int, "torch.cuda.Stream"] = {}


def _side_stream(device) -> "torch.cuda.Stream":
    index = device.index if device.index is not None else torch.cuda.current_device()
    if index not in _SIDE_STREAMS:
        _SIDE_STREAMS[index] = torch.cuda.Stream(device)
    return _SIDE_STREAMS[index]


@register_part("mixer", "parallel_mixers")
class ParallelMixers(Mixer):
    graph_safe = True

    def __init__(self, mixer_left: Mixer, mixer_right: Mixer, left_scale: float = 1.0, right_scale: float = 1.0):
        left, right = mixer_left, mixer_right
        if not getattr(left, "values_are_keys", False) or not hasattr(right, "mix_projected") or left.hidden_size != right.hidden_size:
            raise ValueError("side by side stand attention whose values are its keys (left) and a matrix memory (right) of one width")
        if left.has_out_bias:
            raise ValueError("mixers side by side are not built with a bias of the output projection")
        self.left, self.right = left, right
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        # the block multiplies by the left factor; a left factor of zero leaves the right mixer alone
        self.out_scale = self.left_scale if self.left_scale != 0.0 else 1.0
        self.right_factor = self.right_scale / self.out_scale
        self._in: Optional[torch.Tensor] = None
        self._in_bias: Optional[torch.Tensor] = None
        self._out: Optional[torch.Tensor] = None
        self.out_pad = 0

    def cache_spec(self) -> Optional[KVCacheSpec]:
        return self.left.cache_spec()

    def state_spec(self) -> Optional[StateSpec]:
        return self.right.state_spec()

    def activation_width(self) -> int:
        return self.left.activation_width() + self.right.activation_width() + self.left.hidden_size

    def prepare(self, dtype, device) -> None:
        L, R = self.left, self.right
        if self._in is not None and self._in.device == L.qkv.device and L.qkv.data_ptr() == self._in.data_ptr():
            return
        rows = L.qkv.shape[0] + R.in_proj.shape[0]
        pad = -rows % 16                                   # what the weight-streaming product with a cache write takes
        self._in = torch.cat([L.qkv, R.in_proj, L.qkv.new_zeros((pad, L.qkv.shape[1]))], 0).contiguous()
        self._in_bias = None
        if L.qkv_bias is not None:
            self._in_bias = torch.cat([L.qkv_bias, L.qkv_bias.new_zeros(rows + pad - L.qkv_bias.shape[0])], 0).contiguous()
        left_o = L.o if self.left_scale != 0.0 else torch.zeros_like(L.o)
        self.out_pad = -(L.o.shape[1] + R.o.shape[1]) % 8
        self._out = torch.cat([left_o, R.o, L.o.new_zeros((L.o.shape[0], self.out_pad))], 1).contiguous()
        # the parts' own matrices become views of the merged ones
        n = L.qkv.shape[0]
        L.qkv, R.in_proj = self._in[:n], self._in[n:rows]
        if self.left_scale != 0.0:
            L.o = self._out[:, :L.o.shape[1]]
        R.o = self._out[:, L.o.shape[1]:L.o.shape[1] + R.o.shape[1]]

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        L, R = self.left, self.right
        a, b = L.q_size, R.v_size
        p, cached = L.project(ctx, h, self._in, self._in_bias, cache)
        make = torch.zeros if self.out_pad else torch.empty
        y = make((ctx.n_tokens, a + b + self.out_pad), dtype=p.dtype, device=p.device)
        L.attend_projected(ctx, p, cached, cache, y[:, :a])
        n = L.q_size + L.kv_size
        R.mix_projected(ctx, p[:, n:n + R.in_size], cache, y[:, a:a + b], self.right_factor)
        return matmul_tn(y, self._out)


@register_part("mixer", "normed_parallel_mixers")
class NormedParallelMixers(Mixer):
    graph_safe = True
    emits_pair = True

    def __init__(self, mixer_left: Mixer, mixer_right: Mixer, eps: float, factor: float = 0.5):
        left, right = mixer_left, mixer_right
        if not getattr(left, "qk_filter_taps", 0) or not hasattr(right, "state_floats") or not hasattr(right, "mix_projected") \
                or left.hidden_size != right.hidden_size:
            raise ValueError("side by side stand attention with filtered queries and keys (left) and a selective state space (right) of one width")
        if left.has_out_bias:
            raise ValueError("mixers side by side are not built with a bias of the output projection")
        self.left, self.right = left, right
        self.hidden_size, self.eps, self.factor = left.hidden_size, float(eps), float(factor)
        self.left_at = (right.state_floats() + 3) // 4 * 4          # where a slot's left part starts (16-byte aligned)
        self.left_norm: Optional[torch.Tensor] = None
        self.right_norm: Optional[torch.Tensor] = None
        self._w_left: Optional[torch.Tensor] = None
        self._w_right: Optional[torch.Tensor] = None
        self._in: Optional[torch.Tensor] = None
        self._in_bias: Optional[torch.Tensor] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {n: WeightSpec([(self.hidden_size,)], keep_fp32=True) for n in ("left_norm", "right_norm")}

    def cache_spec(self) -> Optional[KVCacheSpec]:
        return self.left.cache_spec()

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec(((self.left_at + self.left.filter_state_floats() + 3) // 4 * 4,))

    def activation_width(self) -> int:
        return self.left.activation_width() + self.right.activation_width() + 2 * self.hidden_size

    def prepare(self, dtype, device) -> None:
        self._w_left, self._w_right = self.left_norm.float().contiguous(), self.right_norm.float().contiguous()
        L, R = self.left, self.right
        if self._in is not None and self._in.device == L.qkv.device and L.qkv.data_ptr() == self._in.data_ptr():
            return
        n, rows = L.qkv.shape[0], L.qkv.shape[0] + R.in_proj.shape[0]
        pad = -rows % 16                                   # rows of the product stay 16-byte aligned
        self._in = torch.cat([L.qkv, R.in_proj, L.qkv.new_zeros((pad, L.qkv.shape[1]))], 0).contiguous()
        self._in_bias = None
        if L.qkv_bias is not None:
            self._in_bias = torch.cat([L.qkv_bias, L.qkv_bias.new_zeros(rows + pad - n)], 0).contiguous()
        L.qkv, R.in_proj = self._in[:n], self._in[n:rows]  # the parts' own matrices become views of the merged one

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: LayerCache) -> BranchPair:
        L, R = self.left, self.right
        n = L.q_size + L.kv_size
        p = matmul_tn(h, self._in, bias=self._in_bias)
        a = torch.empty((ctx.n_tokens, L.q_size), dtype=p.dtype, device=p.device)
        b = torch.empty((ctx.n_tokens, R.inner), dtype=p.dtype, device=p.device)
        # The halves share nothing but what they read.  A step of single tokens leaves most of the device idle in each of their
        # kernels, so the right one runs on a stream of its own (in a captured step: a branch of the graph); prompt portions fill
        # the device and stay on one stream.
        here = torch.cuda.current_stream(p.device) if CONCURRENT and ctx.decode_only else None
        side = _side_stream(p.device) if here is not None else None
        if side is None:
            R.mix_projected(ctx, p[:, n:n + R.in_size], cache, b)
            y = matmul_tn(b, R.o)
        else:
            side.wait_stream(here)
            with torch.cuda.stream(side):
                R.mix_projected(ctx, p[:, n:n + R.in_size], cache, b)
                y = matmul_tn(b, R.o)
        L.attend_filtered(ctx, p[:, :n], cache, a, self.left_at)
        x = matmul_tn(a, L.o)
        if side is not None:
            here.wait_stream(side)      # before anything that either stream made is read, or given back, by the other
        return BranchPair(x, y, self._w_left, self._w_right, self.eps, self.factor)
