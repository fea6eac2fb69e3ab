"""What happens to the residual stream ahead of a layer run.

``mix_first`` lets the stream meet the embedding output again: x <- W [x; x0],
x0 being the stream as the embedding left it, and (optional) a learned vector of
the turn is added, x <- x + step[t]. A model whose layers run several times in a
row does this once per pass, so that a pass knows which one it is. The product's
result is the new stream (float32); the vector rides into the next layer's first
kernel as what is still to be added to every row.

``add_first`` adds the embedding output to the stream, x <- x + x0, with what is
still pending in the same pass: the sum rides into the next layer's first kernel
as a third summand."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config.spec import PartSpec
from .block import PairSum
from .linear import Linear
from .registry import Runtime, WeightStore, register_part, settle


class MixFirst:
    kind = "mix_first"

    def __init__(self, spec: PartSpec, weights: WeightStore, runtime: Runtime):
        hidden = spec["hidden_size"]
        weight = weights.take(spec["weight"])
        if tuple(weight.shape) != (hidden, 2 * hidden):
            raise ValueError(f"{spec['weight']} is {tuple(weight.shape)}, expected {(hidden, 2 * hidden)}")
        self.mix = Linear(weight, runtime)
        self.steps: Optional[torch.Tensor] = None
        if spec.get("steps"):
            steps = weights.take(spec["steps"])
            if tuple(steps.shape) != (spec["turns"], hidden):
                raise ValueError(f"{spec['steps']} is {tuple(steps.shape)}, expected {(spec['turns'], hidden)}")
            self.steps = steps.to(device=runtime.device, dtype=torch.float32).contiguous()
        self.dtype = runtime.dtype

    def forward(self, residual: torch.Tensor, pending, first: torch.Tensor, turn: int):
        """(new stream, what is to be added to it): ``residual`` with ``pending``
        still to join, ``first`` the embedding output."""
        if pending is not None and not (isinstance(pending, torch.Tensor) and pending.dim() == 2):
            settle(residual, pending)      # anything but a plain result joins the stream first
            pending = None
        mixed = self.mix.forward(ops.join_rows(residual, pending, first, self.dtype), out_dtype=torch.float32)
        return mixed, self.steps[turn] if self.steps is not None else None

    def weight_bytes(self) -> int:
        return self.mix.weight_bytes()


class AddFirst:
    kind = "add_first"

    def __init__(self, spec: PartSpec, weights: WeightStore, runtime: Runtime):
        pass

    def forward(self, residual: torch.Tensor, pending, first: torch.Tensor, turn: int):
        if first.data_ptr() == residual.data_ptr():      # the stream is still the embedding output itself
            residual = residual.clone()
        if isinstance(pending, PairSum) and pending.extra is None:
            return residual, PairSum(pending.first, pending.second, pending.scale, extra=first)
        settle(residual, pending)
        return residual, PairSum(None, None, 1.0, extra=first)

    def weight_bytes(self) -> int:
        return 0


register_part("join", "add_first", lambda spec, weights, runtime: AddFirst(spec, weights, runtime))
register_part("join", "mix_first", lambda spec, weights, runtime: MixFirst(spec, weights, runtime))
