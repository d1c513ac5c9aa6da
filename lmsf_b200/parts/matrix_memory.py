"""A matrix memory with exponential gates (the mLSTM cell of xLSTM): a recurrent mixer whose per-request state is, per head, a
matrix [dk, dv], a vector [dk] and a running maximum, kept in float32 in a state slot (csrc/matrix_memory.cu).

  q = h Wq^T dk^(-1/2), k = h Wk^T  [heads x dk];  v = h Wv^T  [heads x dv]
  i = cap tanh((h Wi^T + bi) / cap);  f = log sigmoid(cap tanh((h Wf^T + bf) / cap))          (one number each per head)
  m_t = max(f + m_(t-1), i);  S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T;  n_t likewise with k alone
  o = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)
  out = (norm_head(o) * w * sigmoid(h Wg^T)) Wo^T                     (the norm per head, its weight over all heads)

q, k, v, the output gate and the two gates' logits come from one merged product.  Gates, state, o and the norm are float32.
Single tokens and short portions are scanned token by token; portions of LONG_PORTION tokens and more are cut into chunks that
run in parallel.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels
from .base import LayerCache, Mixer, StateSpec, StepContext, WeightSpec, register_part
from .linear import matmul_tn

LONG_PORTION = 64      # tokens from which a request's portion is cut into chunks that run in parallel


@register_part("mixer", "matrix_memory")
class MatrixMemory(Mixer):
    graph_safe = True      # every index comes from device tensors; a decode step's launch depends on the batch's size only

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, gate_cap: float, eps: float,
                 floor_eps: float = 1e-6):
        if not (0 < head_dim <= kernels.MEMORY_MAX_DK):
            raise ValueError(f"head_dim {head_dim} is beyond the scan kernel (up to {kernels.MEMORY_MAX_DK})")
        if not gate_cap > 0:
            raise ValueError(f"the gates' cap must be positive, got {gate_cap}")
        self.hidden_size, self.num_heads, self.head_dim, self.value_dim = int(hidden_size), int(num_heads), int(head_dim), int(value_dim)
        self.gate_cap, self.eps, self.floor_eps = float(gate_cap), float(eps), float(floor_eps)
        self.qk_size, self.v_size = self.num_heads * self.head_dim, self.num_heads * self.value_dim
        self.in_size = 2 * self.qk_size + 2 * self.v_size + 2 * self.num_heads
        self.in_proj = self.i_bias = self.f_bias = self.norm = self.o = None
        self._f32: Dict[str, torch.Tensor] = {}

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, H, QK, V = self.hidden_size, self.num_heads, self.qk_size, self.v_size
        return {"in_proj": WeightSpec([(QK, D), (QK, D), (V, D), (V, D), (H, D), (H, D)]),      # q, k, v, gate, i, f
                "i_bias": WeightSpec([(H,)], keep_fp32=True), "f_bias": WeightSpec([(H,)], keep_fp32=True),
                "norm": WeightSpec([(V,)], keep_fp32=True), "o": WeightSpec([(D, V)])}

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((kernels.matrix_memory_state_floats(self.num_heads, self.head_dim, self.value_dim),))

    def activation_width(self) -> int:
        # the product, o in float32 (two), the gated norm; a chunk of 64 tokens keeps a state and a score matrix in float32
        per_chunk = self.num_heads * self.head_dim * (self.value_dim + 1) + self.num_heads * 64 * 64
        return self.in_size + 3 * self.v_size + 2 * (per_chunk // 64)

    def prepare(self, dtype, device) -> None:
        self._f32 = {n: getattr(self, n).float().contiguous() for n in ("i_bias", "f_bias", "norm")}

    @staticmethod
    def _plan(ctx: StepContext):
        """None when no request brings a long portion.  Else (short, chunks, spans, last), made once a step from the host's
        copy of the portions' lengths and shared by all layers: `short` lists the requests that are scanned token by token
        (None if there are none), `chunks` cuts every long portion, `spans` names each portion's chunks, `last` marks its last."""
        if not ctx.q_lens or max(ctx.q_lens) < LONG_PORTION:
            return None
        plan = ctx.extras.get("matrix_memory_plan")
        if plan is None:
            size = kernels.matrix_memory_chunk_tokens()
            short, chunks, spans, last, t0 = [], [], [], [], 0
            for s, n in enumerate(ctx.q_lens):
                if n >= LONG_PORTION:
                    first = len(chunks)
                    for c in range(t0, t0 + n, size):
                        chunks.append((s, c, min(c + size, t0 + n), len(chunks)))
                        last.append(0)
                    last[-1] = 1
                    spans.append((s, first, len(chunks), 0))
                else:
                    short.append((s, t0, t0 + n, 0))
                t0 += n
            rows = short + chunks + spans
            flat = torch.tensor([v for r in rows for v in r] + last, dtype=torch.int32).to(ctx.device, non_blocking=True)
            table, a, b = flat[:4 * len(rows)].view(-1, 4), len(short), len(short) + len(chunks)
            plan = ctx.extras["matrix_memory_plan"] = (table[:a] if a else None, table[a:b], table[b:], flat[4 * len(rows):])
        return plan

    def mix_projected(self, ctx: StepContext, p: torch.Tensor, cache: LayerCache, out: torch.Tensor, out_scale: float = 1.0) -> None:
        """From the rows of the merged product (a view [n, in_size]) to what the output projection reads, times out_scale, in
        `out` (a view [n, v_size])."""
        a, b, H = self.qk_size, self.v_size, self.num_heads
        q, k, v, g = p[:, :a], p[:, a:2 * a], p[:, 2 * a:2 * a + b], p[:, 2 * a + b:2 * a + 2 * b]
        gi, gf = p[:, 2 * (a + b):2 * (a + b) + H], p[:, 2 * (a + b) + H:2 * (a + b) + 2 * H]
        o = torch.empty((ctx.n_tokens, b), dtype=torch.float32, device=p.device)
        w = self._f32
        args = (o, q, k, v, gi, gf, w["i_bias"], w["f_bias"], cache.state, ctx.cu_q, ctx.state_slot, ctx.n_seqs, H, self.head_dim,
                self.value_dim, self.gate_cap, self.head_dim ** -0.5, self.floor_eps)
        plan = self._plan(ctx)
        if plan is None:
            kernels.matrix_memory(*args)
        else:
            short, chunks, spans, last = plan
            if short is not None:
                kernels.matrix_memory(*args, items=short)
            kernels.matrix_memory(*args, items=chunks, spans=spans, last_chunk=last)
        kernels.grouped_gated_norm(out, o, g, w["norm"], self.value_dim, self.eps, gate_act="sigmoid", out_scale=out_scale)

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        p = matmul_tn(h, self.in_proj)
        y = torch.empty((ctx.n_tokens, self.v_size), dtype=p.dtype, device=p.device)
        self.mix_projected(ctx, p, cache, y)
        return matmul_tn(y, self.o)
