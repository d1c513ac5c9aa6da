"""A gated recurrence element by element whose gates read the current token only (minGRU): a recurrent mixer whose per-request
state is one float32 value per channel (csrc/min_gru.cu).

  z = sigmoid(h Wz^T + bz);  u = h Wx^T + bx;  candidate = u + 1/2 where u >= 0, sigmoid(u) elsewhere
  S_t = (1 - z) S_(t-1) + z candidate;   out = (S_t * silu(h Wg^T)) Wo^T

The three projections are one merged product; gates, candidate and state are float32.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels
from .base import LayerCache, Mixer, StateSpec, StepContext, WeightSpec, register_part
from .linear import matmul_tn


@register_part("mixer", "min_gru")
class MinGRU(Mixer):
    graph_safe = True

    def __init__(self, hidden_size: int, width: int):
        self.hidden_size, self.width = int(hidden_size), int(width)
        self.zxg: Optional[torch.Tensor] = None
        self.z_bias: Optional[torch.Tensor] = None
        self.x_bias: Optional[torch.Tensor] = None
        self.o: Optional[torch.Tensor] = None
        self._bz: Optional[torch.Tensor] = None
        self._bx: Optional[torch.Tensor] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {"zxg": WeightSpec([(self.width, self.hidden_size)] * 3),
                "z_bias": WeightSpec([(self.width,)], keep_fp32=True), "x_bias": WeightSpec([(self.width,)], keep_fp32=True),
                "o": WeightSpec([(self.hidden_size, self.width)])}

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self.width,))

    def activation_width(self) -> int:
        return 4 * self.width

    def prepare(self, dtype, device) -> None:
        self._bz, self._bx = self.z_bias.float().contiguous(), self.x_bias.float().contiguous()

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        w = self.width
        p = matmul_tn(h, self.zxg)
        y = torch.empty((ctx.n_tokens, w), dtype=p.dtype, device=p.device)
        kernels.min_gru(y, p[:, :w], p[:, w:2 * w], p[:, 2 * w:], self._bz, self._bx, cache.state, ctx.cu_q, ctx.state_slot,
                        ctx.n_seqs, ctx.max_q_len)
        return matmul_tn(y, self.o)
