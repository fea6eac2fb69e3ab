"""Two mixers side by side: both read the same input, each keeps what it
needs in a cache entry of its own, and the result is
left_scale * left + right_scale * right (summed in float32).

With ``left_norm`` and ``right_norm`` each output passes an RMS norm of its own
first. The pair is then handed on as it is (``NormedPair``): both norms, the
weighted sum, the residual sum and the next sublayer's norm are one kernel."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..config.spec import CacheNeed, PartSpec
from .norm import RMSNorm
from .registry import CacheView, Runtime, StepContext, WeightStore, build_part, graph_safe, register_part


@dataclass
class NormedPair:
    """x += a * norm_l(left + left_bias) + b * norm_r(right), on its way into the residual stream. ``left`` may be
    float32 ``[parts, rows, size]`` summands."""

    left: torch.Tensor
    right: torch.Tensor
    left_norm: RMSNorm
    right_norm: RMSNorm
    weights: tuple
    left_bias: Optional[torch.Tensor] = None

    def _add(self, residual: torch.Tensor, **norm):
        return ops.pair_norm(residual, self.left, self.right, self.left_norm.weight, self.right_norm.weight,
                             self.left_norm.eps, self.right_norm.eps, *self.weights, left_bias=self.left_bias, **norm)

    def settle(self, residual: torch.Tensor) -> None:
        self._add(residual)

    def settle_and_norm(self, residual: torch.Tensor, weight: torch.Tensor, eps: float, out_dtype: torch.dtype) -> torch.Tensor:
        return self._add(residual, weight=weight, eps=eps, out_dtype=out_dtype)


class ParallelMixers:
    kind = "parallel_mixers"

    def __init__(self, spec: PartSpec, weights: WeightStore, runtime: Runtime):
        self.left = build_part("mixer", spec["left"], weights, runtime)
        self.right = build_part("mixer", spec["right"], weights, runtime)
        self.left_scale, self.right_scale = float(spec["left_scale"]), float(spec["right_scale"])
        self.graph_safe = graph_safe(self.left) and graph_safe(self.right)
        self.left_norm = build_part("norm", spec.get("left_norm"), weights, runtime)
        self.right_norm = build_part("norm", spec.get("right_norm"), weights, runtime)
        for norm in (self.left_norm, self.right_norm):
            if (norm is None) != (self.left_norm is None) or (norm is not None and not isinstance(norm, RMSNorm)):
                raise ValueError("both outputs pass an RMS norm, or neither does")
        self.leaves_pending = self.left_norm is not None      # forward_pending is the way to run it

    def parts(self):
        return [self.left, self.right, self.left_norm, self.right_norm]

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kind="several", members=(self.left.cache_need(), self.right.cache_need()))

    def forward_pair(self, x: torch.Tensor, ctx: StepContext, cache: CacheView):
        """(left result, right result, (left_scale, right_scale)) for a caller
        that adds them up itself in a pass it makes anyway."""
        if len(cache.members) != 2:
            raise ValueError("two mixers side by side need a cache view with two members")
        left = self.left.forward(x, ctx, cache.members[0])
        right = self.right.forward(x, ctx, cache.members[1])
        return left, right, (self.left_scale, self.right_scale)

    def forward_pending(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> NormedPair:
        if len(cache.members) != 2:
            raise ValueError("two mixers side by side need a cache view with two members")
        bias = getattr(self.left, "out_bias", None)
        run = getattr(self.left, "forward_unbiased", self.left.forward)     # the pair's kernel adds the bias and summands
        return NormedPair(run(x, ctx, cache.members[0]), self.right.forward(x, ctx, cache.members[1]), self.left_norm,
                          self.right_norm, (self.left_scale, self.right_scale), bias)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> torch.Tensor:
        if self.leaves_pending:
            out = torch.zeros(x.shape, dtype=torch.float32, device=x.device)
            self.forward_pending(x, ctx, cache).settle(out)
            return out
        left, right, (a, b) = self.forward_pair(x, ctx, cache)
        return ops.weighted_sum(left, right, a, b)

    def weight_bytes(self) -> int:
        return self.left.weight_bytes() + self.right.weight_bytes()


register_part("mixer", "parallel_mixers", lambda spec, weights, runtime: ParallelMixers(spec, weights, runtime))
