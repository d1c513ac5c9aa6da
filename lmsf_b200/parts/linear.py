"""Dense projections y = x W^T (+ b where the model has biases), weight stored [out, in] as in the checkpoint.

The reference's linear family (core/src/model_executor/layers/linear.rs:28-106, :325-497, :499-728)
wraps cuBLASLt and merges q, k, v (and gate, up) into one matrix by row ranges; the same merged
layouts are used here.  bfloat16 products of more than 16 rows go to the library (cuBLAS through torch.mm),
the place where the reference calls a library too; products of up to 16 rows (decode steps) run on
this package's weight-streaming kernel (csrc/gemm_skinny.cu); float32 products run on this package's own FFMA kernel so
that no reduced-precision mode can slip in and a row's result does not depend on the batch.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence, Union

import torch

from .. import kernels
from .base import NormAfter, Part, Prenormed, WeightSpec, register_part

# Library products must add up in float32: with torch's default a split-k bfloat16 product may add its partial sums
# in bfloat16, and a row's result would then depend on how many rows share the product (on how a prompt was cut).
torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False

_MM_HAS_OUT_DTYPE: Optional[bool] = None
USE_SKINNY = True     # bfloat16 products of up to 16 rows run on this package's weight-streaming kernel
SKINNY_TALL_FROM = 65536   # ... except 9 to 16 rows against this many output features and more


def _skinny_takes(x: torch.Tensor, w: torch.Tensor) -> bool:
    # (9 to 16 rows against a very tall matrix, the head: a stage of the kernel then holds as much of x as of w, and the
    # library is faster: 162 against 182 us for 128,256 x 4,096 at 16 rows)
    return USE_SKINNY and kernels.gemm_skinny_supported(x, w) and not (x.shape[0] > 8 and w.shape[0] >= SKINNY_TALL_FROM)


def matmul_tn(x: Union[torch.Tensor, Prenormed], w: torch.Tensor, out_dtype: Optional[torch.dtype] = None,
              bias: Optional[torch.Tensor] = None, act: Optional[str] = None) -> torch.Tensor:
    """x [M, K] times w [N, K] transposed -> [M, N] in `out_dtype` (default: x's dtype), plus `bias` [N] if given.  The
    bfloat16 products add a bfloat16 bias to their float32 sums before they round (the reference adds it afterwards, in a
    step of its own: layers/linear.rs:100-104); otherwise a kernel adds it after the product.  `act` "relu2": the square of
    max(result, 0).  x may be a `Prenormed`: the weight-streaming kernel divides its sums by the rows' root mean square."""
    plain = not isinstance(x, Prenormed)
    hx = x if plain else x.x
    fused_bias = bias if (bias is not None and bias.dtype == torch.bfloat16 and hx.dtype == torch.bfloat16) else None
    dt = out_dtype or hx.dtype
    if (fused_bias is not None or act is not None) and (bias is None or fused_bias is not None) and _skinny_takes(hx, w) and \
            dt in (torch.bfloat16, torch.float32):
        y = torch.empty((hx.shape[0], w.shape[0]), dtype=dt, device=w.device)
        kernels.gemm_skinny(y, hx, w, prenorm=None if plain else (x.sumsq, x.eps, x.width), bias=fused_bias, act=act)
        return y
    if plain and fused_bias is not None and dt == torch.bfloat16:
        y = torch.addmm(fused_bias, x, w.t())
        if act is not None:
            kernels.relu2_(y)
        return y
    if isinstance(x, Prenormed):
        if _skinny_takes(x.x, w) and dt in (torch.bfloat16, torch.float32):
            y = torch.empty((x.x.shape[0], w.shape[0]), dtype=dt, device=w.device)
            kernels.gemm_skinny(y, x.x, w, prenorm=(x.sumsq, x.eps, x.width))
        else:
            y = _product_tn(x.norm.finish(x), w, out_dtype)
    else:
        y = _product_tn(x, w, out_dtype)
    if bias is not None:
        kernels.bias_add(y, bias if bias.dtype == y.dtype else bias.to(y.dtype))
    if act is not None:
        kernels.relu2_(y)
    return y


def _product_tn(x: torch.Tensor, w: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    global _MM_HAS_OUT_DTYPE
    out_dtype = out_dtype or x.dtype
    if x.dtype == torch.float32:
        out = torch.empty((x.shape[0], w.shape[0]), dtype=torch.float32, device=x.device)
        kernels.gemm_tn_simt(out, x, w)
        return out if out_dtype == torch.float32 else out.to(out_dtype)
    if _skinny_takes(x, w) and out_dtype in (torch.bfloat16, torch.float32):
        out = torch.empty((x.shape[0], w.shape[0]), dtype=out_dtype, device=x.device)
        kernels.gemm_skinny(out, x, w)
        return out
    if out_dtype == x.dtype:
        return torch.mm(x, w.t())
    if _MM_HAS_OUT_DTYPE is not False:
        try:
            y = torch.mm(x, w.t(), out_dtype=out_dtype)
            _MM_HAS_OUT_DTYPE = True
            return y
        except (TypeError, RuntimeError):
            if _MM_HAS_OUT_DTYPE:
                raise
            _MM_HAS_OUT_DTYPE = False
    out = torch.empty((x.shape[0], w.shape[0]), dtype=out_dtype, device=x.device)
    kernels.gemm_tn_simt(out, x, w)
    return out


def batched_matmul_tn(out: torch.Tensor, a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """out[:, b, :] = a[:, b, :] w[b]^T for every b: one product per head of an activation matrix.
    a: [M, B, K] and out: [M, B, N] are views with a contiguous last dimension; w: [B, N, K].
    bfloat16 with more than 16 rows: the library's batched product; else this package's FFMA kernel (true 32-bit
    for float32; few rows in bfloat16, where the product is a stream over w)."""
    if a.dtype == torch.bfloat16 and a.shape[0] > kernels.SKINNY_MAX_M:
        torch.bmm(a.transpose(0, 1), w.transpose(1, 2), out=out.transpose(0, 1))
    else:
        kernels.gemm_tn_simt_batched(out, a, w)
    return out


def matmul_tn_residual(x: torch.Tensor, w: torch.Tensor, then: NormAfter) -> Optional[Prenormed]:
    """The product before a norm, for a few rows: then.res += x w^T, and the first half of then.norm on the new
    residual.  None when this product cannot do it (the caller then multiplies as usual and the norm runs whole)."""
    norm, res = then.norm, then.res
    weight = getattr(norm, "weight", None)
    if not (norm.splittable and _skinny_takes(x, w) and weight is not None and res.dtype == torch.float32
            and res.shape == (x.shape[0], w.shape[0]) and res.is_contiguous() and weight.shape == (w.shape[0],)):
        return None
    parts = kernels.gemm_skinny_residual_parts(w.shape[0])
    sumsq = torch.empty((x.shape[0], (parts + 3) // 4 * 4), dtype=torch.float32, device=x.device)[:, :parts]
    xg = torch.empty((x.shape[0], w.shape[0]), dtype=torch.bfloat16, device=x.device)
    kernels.gemm_skinny_residual(xg, x, w, res, weight, sumsq)
    return Prenormed(xg, sumsq, norm.eps, w.shape[0], norm, res)


@register_part("linear", "dense")
class Linear(Part):
    """out_features may be a list: the sources are stacked along the output dimension."""
    graph_safe = True

    def __init__(self, in_features: int, out_features: Union[int, Sequence[int]], out_dtype: Optional[str] = None,
                 bias: bool = False, out_scale: float = 1.0, out_softcap: Optional[float] = None):
        # an output head may scale its float32 results and cap them smoothly: cap * tanh(scale * y / cap)
        self.out_scale, self.out_softcap = float(out_scale), float(out_softcap or 0.0)
        self.in_features = int(in_features)
        self.has_bias = bool(bias)
        self.bias: Optional[torch.Tensor] = None
        self.out_splits: List[int] = [int(out_features)] if isinstance(out_features, int) else [int(o) for o in out_features]
        self.out_features = sum(self.out_splits)
        self.out_dtype = {None: None, "float32": torch.float32, "bfloat16": torch.bfloat16}[out_dtype]
        self.weight: Optional[torch.Tensor] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        specs = {"weight": WeightSpec([(o, self.in_features) for o in self.out_splits])}
        if self.has_bias:
            specs["bias"] = WeightSpec([(o,) for o in self.out_splits])
        return specs

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        y = matmul_tn(x, self.weight, self.out_dtype, self.bias)
        if self.out_scale != 1.0 or self.out_softcap:
            if y.dtype != torch.float32:
                raise ValueError("a scaled or capped output is float32 (out_dtype='float32')")
            kernels.scale_softcap_(y, self.out_scale, self.out_softcap)
        return y


@register_part("linear", "gate_logits")
class GateLogits(Part):
    """The logits of one or several gates that read the same input: z = x W^T in float32, W the gates' matrices stacked
    along the output dimension, and their biases (kept apart, in float32, for the kernel that applies the sigmoids)."""
    graph_safe = True

    def __init__(self, in_features: int, out_features: Union[int, Sequence[int]], bias: bool = True):
        self.in_features = int(in_features)
        self.out_splits: List[int] = [int(out_features)] if isinstance(out_features, int) else [int(o) for o in out_features]
        self.out_features = sum(self.out_splits)
        self.has_bias = bool(bias)
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None
        self._bias32: Optional[torch.Tensor] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        specs = {"weight": WeightSpec([(o, self.in_features) for o in self.out_splits])}
        if self.has_bias:
            specs["bias"] = WeightSpec([(o,) for o in self.out_splits], keep_fp32=True)
        return specs

    def prepare(self, dtype, device) -> None:
        self._bias32 = self.bias.float().contiguous() if self.has_bias else None

    def bias_f32(self) -> Optional[torch.Tensor]:
        return self._bias32

    def logits(self, x: torch.Tensor) -> torch.Tensor:
        return matmul_tn(x, self.weight, out_dtype=torch.float32)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        z = self.logits(x)
        if self._bias32 is not None:
            kernels.bias_add(z, self._bias32)
        return z
