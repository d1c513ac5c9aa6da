"""What a mixer or a feed-forward reads is mixed with what it would have read some tokens earlier.

Token shift:

  h'_t = h_t + (h_{t-1} - h_t) * mix        (element by element; mix is a learned vector of the stream's width)

h_{t-1} is the row of the token before in the same request as it was BEFORE this replacement, and zeros for the request's
first token.  Between steps it is state of the request (float32 [width] per state slot): a portion's first token reads the
slot, the portion's last row is left there.  One kernel (csrc/stream_norm.cu, `token_shift`), float32 inside.

Filter shift:
  h'_t = h_t + sum_j f[:, j] * h_{t - taps + 1 + j}        (a short causal filter per channel; zeros before the first token)
Its state is the last taps - 1 rows h (float32 [taps - 1, width] per slot).  Prompt portions run on the convolution's kernel
(csrc/recurrent.cu); a step of single tokens may have it done by the kernel that norms the rows (`single_token_filter`).
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels
from .base import Shift, StateSpec, StepContext, WeightSpec, register_part


@register_part("shift", "token_shift")
class TokenShift(Shift):
    graph_safe = True

    def __init__(self, hidden_size: int):
        self.hidden_size = int(hidden_size)
        self.mix: Optional[torch.Tensor] = None
        self._mix32: Optional[torch.Tensor] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {"mix": WeightSpec([(self.hidden_size,)], keep_fp32=True)}

    def state_spec(self) -> StateSpec:
        return StateSpec((self.hidden_size,), torch.float32)

    def prepare(self, dtype, device) -> None:
        self._mix32 = self.mix.float().contiguous()

    def forward(self, ctx: StepContext, h: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
        out = torch.empty_like(h)
        kernels.token_shift(out, h, self._mix32, state, ctx.positions, ctx.token_seq, ctx.cu_q, ctx.state_slot)
        return out


@register_part("shift", "filter_shift")
class FilterShift(Shift):
    graph_safe = True

    def __init__(self, hidden_size: int, taps: int):
        self.hidden_size, self.taps = int(hidden_size), int(taps)
        if not (1 <= self.taps <= kernels.CONV_MAX_TAPS):
            raise ValueError(f"a filter of {taps} taps is beyond the kernel (1 to {kernels.CONV_MAX_TAPS})")
        self.filter: Optional[torch.Tensor] = None
        self._f32: Optional[torch.Tensor] = None
        self._by_tap: Optional[torch.Tensor] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {"filter": WeightSpec([(self.hidden_size, self.taps)], keep_fp32=True)}

    def state_spec(self) -> StateSpec:
        return StateSpec((max(1, self.taps - 1) * self.hidden_size,), torch.float32)

    def prepare(self, dtype, device) -> None:
        self._f32 = self.filter.float().contiguous()
        self._by_tap = self._f32.t().contiguous()

    def activation_width(self) -> int:
        return self.hidden_size

    def single_token_filter(self) -> Optional[torch.Tensor]:
        return self._by_tap

    def forward(self, ctx: StepContext, h: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
        out = torch.empty_like(h)
        kernels.causal_conv(out, h, self._f32, None, state, 0, ctx.cu_q, ctx.state_slot, ctx.n_seqs, max(ctx.max_q_len, 1), act="add_input")
        return out
