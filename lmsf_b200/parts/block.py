"""Arrangements of parts inside one layer.

`pre_norm` is the reference's Block (core/src/model_executor/models/llama/llama.rs:276-385): norm,
mixer, norm, feed-forward, where each residual add is deferred into the following norm
(llama.rs:295-317, :333) and the layer hands (branch output, residual) to the next one.
"""
from __future__ import annotations

import os
from typing import Dict, Optional, Tuple

import torch

from .. import kernels
from .base import Block, BranchPair, LayerCache, Norm, NormAfter, Normed, Part, Shift, StepContext, register_part

# A step of a few tokens in bfloat16: a norm between two weight-streaming products is done by those products
# (the one before adds to the residual stream and leaves sums of squares, the one after divides).  LMSF_FUSE_NORMS=0:
# every norm is a kernel of its own.
FUSE_NORMS = os.environ.get("LMSF_FUSE_NORMS", "1") != "0"


def divides_rows(norm: Optional[Norm]) -> bool:
    """Whether a norm is a division by the root mean square and one weight: what the kernels that end a block apply."""
    return hasattr(norm, "weight_f32") and not norm.centred and not getattr(norm, "has_layer_scale", False)


def norm_after(ctx: StepContext, producer: Part, norm: Norm, consumer: Part, res: Optional[torch.Tensor]) -> Optional[NormAfter]:
    """The offer to `producer` to take `norm` into its last product, if everybody involved is able to on this step."""
    if (FUSE_NORMS and res is not None and getattr(producer, "fuses_norm", False)
            and getattr(consumer, "takes_prenormed", False) and getattr(norm, "splittable", False)
            and ctx.dtype == torch.bfloat16 and ctx.n_tokens <= kernels.SKINNY_MAX_M):
        return NormAfter(norm, res)
    return None


@register_part("block", "pre_norm")
class PreNormBlock(Block):
    ROLES = {"mixer_norm": "norm", "mixer": "mixer", "ffn_norm": "norm", "feed_forward": "feed_forward"}

    def __init__(self, parts: Dict[str, Part]):
        super().__init__(parts)
        self.mixer_norm, self._mixer = parts["mixer_norm"], parts["mixer"]
        self.ffn_norm, self.feed_forward = parts["ffn_norm"], parts["feed_forward"]

    fuses_next_norm = True

    def entry(self) -> Optional[Tuple[Norm, Part]]:
        return self.mixer_norm, self._mixer

    def forward(self, ctx: StepContext, x, res: Optional[torch.Tensor], cache: LayerCache,
                next_entry: Optional[Tuple[Norm, Part]] = None):
        h, res = self.mixer_norm.forward_residual(x, res)
        then = norm_after(ctx, self._mixer, self.ffn_norm, self.feed_forward, res)
        a = self._mixer.forward(ctx, h, cache, then=then) if then is not None else self._mixer.forward(ctx, h, cache)
        h, res = self.ffn_norm.forward_residual(a, res)
        then = norm_after(ctx, self.feed_forward, next_entry[0], next_entry[1], res) if next_entry is not None else None
        out = self.feed_forward.forward(ctx, h, then=then) if then is not None else self.feed_forward.forward(ctx, h)
        return out, res


@register_part("block", "sandwich_norm")
class SandwichNormBlock(Block):
    """A norm before AND after each branch:  x <- x + post(mixer(pre(x))),  x <- x + post(ff(pre(x))), where a post norm
    may carry a layer scale (a learned vector that multiplies its output).  The residual stream is float32 and every
    sum into it is made in float32 from the float32 normed branch (the branch is never rounded before it is added).
    One kernel does what lies between two branches: the post norm of the branch before, the add, and the pre norm of
    the branch after (`kernels.stream_norm`, or `kernels.stream_layer` where a norm takes the mean off); with `next_entry` it
    also applies the next block's first norm and hands it over as a `Normed`.  A layer may have no feed-forward.  With a
    `mixer_shift` or a `ffn_shift` the mixer or the feed-forward reads its norm's output mixed with rows of the tokens before (a
    `Shift` part, whose state per request the block declares); in a step of single tokens a shift that is a short filter is part
    of the kernel that norms the rows.  A mixer may return a `BranchPair`, which the same kernel joins."""
    ROLES = {"mixer_norm": "norm", "mixer_shift": "shift", "mixer": "mixer", "mixer_post_norm": "norm",
             "ffn_norm": "norm", "ffn_shift": "shift", "feed_forward": "feed_forward", "ffn_post_norm": "norm"}
    OPTIONAL_ROLES = ("mixer_shift", "ffn_norm", "ffn_shift", "feed_forward", "ffn_post_norm")
    fuses_next_norm = True
    fuses_next_shift = True
    takes_pair = True

    def __init__(self, parts: Dict[str, Part]):
        super().__init__(parts)
        self.mixer_norm, self._mixer, self.mixer_post = parts["mixer_norm"], parts["mixer"], parts["mixer_post_norm"]
        self.mixer_shift, self.ffn_shift = parts.get("mixer_shift"), parts.get("ffn_shift")
        self.feed_forward = parts.get("feed_forward")
        self.ffn_norm, self.ffn_post = parts.get("ffn_norm"), parts.get("ffn_post_norm")
        if self.feed_forward is not None and (self.ffn_norm is None or self.ffn_post is None):
            raise ValueError("a feed-forward needs the norms before and after it")
        for n in (self.mixer_norm, self.mixer_post, self.ffn_norm, self.ffn_post):
            if n is not None and not hasattr(n, "weight_f32"):
                raise ValueError("the sandwich block takes norms that are a factor per row times a weight (rmsnorm, layernorm)")

    def entry(self) -> Optional[Tuple[Norm, Part]]:
        return self.mixer_norm, self._mixer

    def entry_shift(self) -> Optional[Shift]:
        return self.mixer_shift

    def state_specs(self):
        return {role: p.state_spec() for role, p in (("mixer_shift", self.mixer_shift), ("ffn_shift", self.ffn_shift)) if p is not None}

    @staticmethod
    def _between(ctx: StepContext, res: torch.Tensor, branch, post: Optional[Norm], nxt: Optional[Norm], shift=None):
        """res += post(branch) (if there is a branch: a tensor or a pair); returns (nxt(res) in the activation type, None without
        nxt; whether it has passed `shift`, a (part, state) behind nxt, as well)."""
        filt = None
        if shift is not None and nxt is not None and FUSE_NORMS and ctx.decode_only and ctx.n_tokens == ctx.n_seqs:
            f = shift[0].single_token_filter()
            filt = (f, shift[1], ctx.state_slot) if f is not None else None
        pair = branch if isinstance(branch, BranchPair) else None
        y = branch.first if pair is not None else branch
        h = torch.empty(res.shape, dtype=ctx.dtype, device=res.device) if nxt is not None else None
        if pair is not None or filt is not None or branch is None or post.centred or (nxt is not None and nxt.centred):
            if post is not None and getattr(post, "has_layer_scale", False):
                raise ValueError("a layer scale is not built with norms that take the mean off, pairs of branches and filters")
            kernels.stream_layer(res, y=y, pair=(pair.second, pair.w_first, pair.w_second, pair.eps, pair.factor) if pair is not None else None,
                                 w_post=post.weight_f32() if y is not None else None, eps_post=post.eps if y is not None else 0.0,
                                 post_centred=y is not None and post.centred, h=h, w_next=nxt.weight_f32() if nxt is not None else None,
                                 eps_next=nxt.eps if nxt is not None else 0.0, next_centred=nxt is not None and nxt.centred, filt=filt)
            return h, filt is not None
        kernels.stream_norm(res, y=branch, w_post=post.weight_f32(), layer_scale=post.scale_f32(), eps_post=post.eps,
                            h=h, w_next=nxt.weight_f32() if nxt is not None else None,
                            eps_next=nxt.eps if nxt is not None else 0.0)
        return h, False

    def forward(self, ctx: StepContext, x, res: Optional[torch.Tensor], cache: LayerCache,
                next_entry: Optional[Tuple[Norm, Part]] = None, next_shift=None):
        own = [(p, cache.extra[role]) if p is not None else None for role, p in (("mixer_shift", self.mixer_shift), ("ffn_shift", self.ffn_shift))]
        if x is None and own[0] is not None and own[0][0].single_token_filter() is not None:      # a complete stream
            h, shifted = self._between(ctx, res, None, None, self.mixer_norm, own[0])
        else:
            shifted = isinstance(x, Normed) and x.shifted
            h, res = self.mixer_norm.forward_residual(x, res)      # x: None (complete stream), a Normed, or a pending branch
        if own[0] is not None and not shifted:
            h = own[0][0].forward(ctx, h, own[0][1])
        a = self._mixer.forward(ctx, h, cache)
        nxt = next_entry[0] if next_entry is not None and hasattr(next_entry[0], "weight_f32") and \
            not getattr(next_entry[0], "has_layer_scale", False) else None
        post = self.mixer_post
        if self.feed_forward is not None:
            h, shifted = self._between(ctx, res, a, post, self.ffn_norm, own[1])
            if own[1] is not None and not shifted:
                h = own[1][0].forward(ctx, h, own[1][1])
            a, post = self.feed_forward.forward(ctx, h), self.ffn_post
        h, shifted = self._between(ctx, res, a, post, nxt, next_shift)
        return (Normed(h, nxt, res, shifted) if nxt is not None else None), res


@register_part("block", "branch_norm")
class BranchNormBlock(Block):
    """Norms on the branches' outputs only:  x <- x + m * norm(mixer(x)),  x <- x + m * norm(ff(x)), and, where the layer
    has one, a third branch after the feed-forward, x <- x + m * norm(side(x)).  The branches read the stream itself (in
    the activation type); m is one factor for the whole model.  The residual stream is float32 and every sum into it is
    made in float32 from the float32 normed branch.  One kernel does what lies between two branches: the norm of the
    branch before, the scaled add, and the stream in the activation type for the branch after (`kernels.stream_norm`
    without a next norm); with `next_entry` of a block of this kind the last of them also serves the next block."""
    ROLES = {"mixer": "mixer", "mixer_post_norm": "norm", "feed_forward": "feed_forward", "ffn_post_norm": "norm",
             "side": "feed_forward", "side_post_norm": "norm"}
    OPTIONAL_ROLES = ("feed_forward", "ffn_post_norm", "side", "side_post_norm")
    fuses_next_norm = True

    def __init__(self, parts: Dict[str, Part], residual_mult: float = 1.0):
        super().__init__(parts)
        self.residual_mult = float(residual_mult)
        self._mixer = parts["mixer"]
        self.branches = [(parts["mixer"], parts["mixer_post_norm"])]
        for role, norm in (("feed_forward", "ffn_post_norm"), ("side", "side_post_norm")):
            if role in parts:
                if norm not in parts:
                    raise ValueError(f"the branch {role!r} needs its norm {norm!r}")
                self.branches.append((parts[role], parts[norm]))
        for _, n in self.branches:
            if not divides_rows(n):
                raise ValueError("the branch-norm block takes norms that are a factor per row times a weight (rmsnorm)")

    def entry(self) -> Optional[Tuple[Norm, Part]]:
        return None, self._mixer          # no norm before the first branch: it wants the stream itself

    def forward(self, ctx: StepContext, x, res: Optional[torch.Tensor], cache: LayerCache,
                next_entry: Optional[Tuple[Norm, Part]] = None):
        if isinstance(x, Normed):             # the block before left the stream in the activation type
            if x.norm is not None or x.res is not res:
                raise ValueError("a prepared activation was made for another norm or residual stream")
            h = x.h
        elif x is None:                       # a complete float32 stream
            h = self._as_activation(ctx, res)
        elif res is None:                     # the embedding's output starts the stream
            h = x
            if x.dtype == torch.float32:
                res = x
            else:
                res = torch.empty(x.shape, dtype=torch.float32, device=x.device)
                kernels.stream_begin(res, x)
        else:
            raise ValueError("the branch-norm block takes a complete stream, not a pending branch")
        wants_stream = next_entry is not None and next_entry[0] is None
        for i, (part, norm) in enumerate(self.branches):
            y = part.forward(ctx, h, cache) if i == 0 else part.forward(ctx, h)
            last = i == len(self.branches) - 1
            need_h = (not last) or wants_stream
            h = torch.empty_like(y) if (need_h and ctx.dtype != torch.float32) else None
            kernels.stream_norm(res, y=y, w_post=norm.weight_f32(), eps_post=norm.eps, h=h,
                                branch_scale=self.residual_mult)
            if need_h and h is None:
                h = res                       # float32 activations: the stream itself (no part writes its input)
        return (Normed(h, None, res) if wants_stream else None), res

    @staticmethod
    def _as_activation(ctx: StepContext, res: torch.Tensor) -> torch.Tensor:
        if ctx.dtype == torch.float32:
            return res
        h = torch.empty(res.shape, dtype=ctx.dtype, device=res.device)
        kernels.stream_norm(res, h=h)
        return h


@register_part("block", "parallel_gated")
class ParallelGatedBlock(Block):
    """One norm, two branches side by side, each behind a gate of its own:
         h = norm(x);  x <- x + sigmoid(W1 h + b1) * mixer(h) + sigmoid(W2 h + b2) * ff(h)
    The gates are vectors of the stream's width, multiplied element by element; their logits come from ONE product
    (`gates`: a `gate_logits` part whose matrix stacks W1 and W2) in float32.  One kernel ends the layer: both sigmoids,
    both products, the float32 sum into the stream and, when the next block starts with a norm of the same kind, that
    norm too (`kernels.gated_branches`).  A layer may have no feed-forward (and then no second gate)."""
    ROLES = {"norm": "norm", "mixer": "mixer", "feed_forward": "feed_forward", "gates": "linear"}
    OPTIONAL_ROLES = ("feed_forward",)
    fuses_next_norm = True

    def __init__(self, parts: Dict[str, Part]):
        super().__init__(parts)
        self.norm, self._mixer, self.gates = parts["norm"], parts["mixer"], parts["gates"]
        self.feed_forward = parts.get("feed_forward")
        if not divides_rows(self.norm):
            raise ValueError("the parallel block takes a norm that is a factor per row times a weight (rmsnorm)")
        branches = 2 if self.feed_forward is not None else 1
        if not hasattr(self.gates, "logits") or self.gates.out_features != branches * self.norm.hidden_size:
            raise ValueError(f"the parallel block needs gate logits of {branches} x the stream's width")

    def entry(self) -> Optional[Tuple[Norm, Part]]:
        return self.norm, self._mixer

    def forward(self, ctx: StepContext, x, res: Optional[torch.Tensor], cache: LayerCache,
                next_entry: Optional[Tuple[Norm, Part]] = None):
        if x is not None and not isinstance(x, Normed) and res is None:      # the embedding's output starts the stream
            if x.dtype == torch.float32:
                res = x
            else:
                res = torch.empty(x.shape, dtype=torch.float32, device=x.device)
                kernels.stream_begin(res, x)
            x = None
        h, res = self.norm.forward_residual(x, res)       # x: None (a complete stream), a Normed, or a pending branch
        z = self.gates.logits(h)
        a = self._mixer.forward(ctx, h, cache)
        f = self.feed_forward.forward(ctx, h) if self.feed_forward is not None else None
        nxt = next_entry[0] if next_entry is not None and divides_rows(next_entry[0]) else None
        h_next = torch.empty_like(a) if nxt is not None else None
        kernels.gated_branches(res, z, self.gates.bias_f32(), a, f, h=h_next,
                               w_next=nxt.weight_f32() if nxt is not None else None,
                               eps_next=nxt.eps if nxt is not None else 0.0)
        return (Normed(h_next, nxt, res) if nxt is not None else None), res


@register_part("block", "parallel_norms")
class ParallelNormsBlock(Block):
    """Two branches side by side, each behind a norm of its own over the same stream:
         x <- x + (mixer(norm1(x)) + ff(norm2(x)))
    The norms share the root of the mean square, so one kernel ends a layer: both branches' sum into the float32 stream and,
    when the next block is of this kind, both of its norms (`kernels.stream_branches`).  The mixer's output is multiplied by
    its `out_scale` there, in float32.  A layer may have no feed-forward (and then no second norm)."""
    ROLES = {"mixer_norm": "norm", "mixer": "mixer", "ffn_norm": "norm", "feed_forward": "feed_forward"}
    OPTIONAL_ROLES = ("ffn_norm", "feed_forward")
    fuses_next_norm = True
    scales_mixer = True

    def __init__(self, parts: Dict[str, Part]):
        super().__init__(parts)
        self.mixer_norm, self._mixer = parts["mixer_norm"], parts["mixer"]
        self.ffn_norm, self.feed_forward = parts.get("ffn_norm"), parts.get("feed_forward")
        if (self.feed_forward is None) != (self.ffn_norm is None):
            raise ValueError("a feed-forward and its norm go together")
        for n in (self.mixer_norm, self.ffn_norm):
            if n is not None and not divides_rows(n):
                raise ValueError("the block takes norms that are a factor per row times a weight (rmsnorm)")
        if self.ffn_norm is not None and self.ffn_norm.eps != self.mixer_norm.eps:
            raise ValueError("the block's two norms share one eps")

    def entry(self) -> Optional[Tuple[Norm, Part]]:
        return ParallelNorms(self.mixer_norm, self.ffn_norm), self._mixer

    @staticmethod
    def _end(ctx: StepContext, res: torch.Tensor, a, c: float, f, norms: Optional["ParallelNorms"]):
        """res += c * a + f; the two normed forms of it that `norms` asks for."""
        h1 = h2 = None
        if norms is not None:
            h1 = torch.empty(res.shape, dtype=ctx.dtype, device=res.device)
            h2 = torch.empty_like(h1) if norms.second is not None else None
        kernels.stream_branches(res, a, c, f, 1.0, h1, norms.first.weight_f32() if norms is not None else None, h2,
                                norms.second.weight_f32() if h2 is not None else None,
                                norms.first.eps if norms is not None else 0.0)
        return h1, h2

    def forward(self, ctx: StepContext, x, res: Optional[torch.Tensor], cache: LayerCache,
                next_entry: Optional[Tuple[Norm, Part]] = None):
        if isinstance(x, Normed):
            if not isinstance(x.norm, ParallelNorms) or x.norm.first is not self.mixer_norm or x.res is not res:
                raise ValueError("a prepared activation was made for other norms or another residual stream")
            h1, h2 = x.h
        else:
            if x is not None and res is None:       # the embedding's output starts the stream
                res = x if x.dtype == torch.float32 else torch.empty(x.shape, dtype=torch.float32, device=x.device)
                if res is not x:
                    kernels.stream_begin(res, x)
                x = None
            h1, h2 = self._end(ctx, res, x, 1.0, None, ParallelNorms(self.mixer_norm, self.ffn_norm))
        a = self._mixer.forward(ctx, h1, cache)
        f = self.feed_forward.forward(ctx, h2) if self.feed_forward is not None else None
        norms = None
        if next_entry is not None:
            n = next_entry[0]
            if isinstance(n, ParallelNorms):
                norms = n
            elif divides_rows(n):
                norms = ParallelNorms(n, None)
        h1, h2 = self._end(ctx, res, a, self._mixer.out_scale, f, norms)
        if norms is None:
            return None, res
        return (Normed((h1, h2), norms, res) if isinstance(next_entry[0], ParallelNorms) else Normed(h1, norms.first, res)), res


class ParallelNorms:
    """The two norms that a parallel-norms block applies to the stream (the second may be missing); what stands for its first
    norm when the block before is asked to apply it."""

    def __init__(self, first: Norm, second: Optional[Norm]):
        self.first, self.second = first, second
