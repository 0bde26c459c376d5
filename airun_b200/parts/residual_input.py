"""A residual stream mixed with the embedding ahead of a pass over layers that run several times.

    x <- M [x; x0] = Mx x + M0 x0              M = [Mx | M0], [H, 2H]; x0 is the embedding's output

The second term is the same in every pass, so it is worked out once a step; a pass runs one H x H product and leaves
the sum with that term to the first norm of the layer that follows.  The residual stream is float32 and stays so: on the
bfloat16 path x (and x0) enter the products as two bfloat16 halves side by side whose sum is x to 16 bits of mantissa,
[hi | lo] against [Mx | Mx], so a pass costs what one product over [x; x0] would and rounds nothing to bfloat16.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from ..weights.loader import WeightSpec
from .base import CastActivations, PostNormWrite, ResidualInput, register_part
from .linear import linear


class MixWithEmbedding(ResidualInput):
    def __init__(self, prefix: str, hidden_size: int, dtype: torch.dtype = torch.bfloat16, device=None):
        """``prefix``: the full name of the matrix's tensor."""
        self.name, self.H, self.dtype, self.device = prefix, int(hidden_size), dtype, device
        self.w_x: Optional[torch.Tensor] = None
        self.w_0: Optional[torch.Tensor] = None

    def weight_specs(self) -> List[WeightSpec]:
        return [WeightSpec(self.name, (self.H, 2 * self.H))]

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        w = tensors.pop(self.name)
        halves = 2 if self.dtype == torch.bfloat16 else 1
        self.w_x = w[:, :self.H].repeat(1, halves).contiguous()
        self.w_0 = w[:, self.H:].repeat(1, halves).contiguous()

    def _operand(self, ctx, x: torch.Tensor, pending: Optional[PostNormWrite] = None) -> torch.Tensor:
        """x, with what is pending carried out on the way, as the products of this part read it."""
        split = self.dtype == torch.bfloat16
        op = ctx.ws.alloc((x.shape[0], (2 if split else 1) * self.H), self.dtype)
        post = pending.norm_args() if pending is not None else {}
        ops.sandwich_norm(x, op, mode=ops.SANDWICH_SPLIT if split else ops.SANDWICH_COPY, write_back=False, **post)
        return op

    def begin(self, ctx, x0: torch.Tensor) -> torch.Tensor:
        term = ctx.ws_main.alloc((x0.shape[0], self.H), torch.float32)
        return linear(ctx, self._operand(ctx, x0), self.w_0, term)

    def forward(self, ctx, x: torch.Tensor, pending, kept: torch.Tensor):
        if isinstance(pending, torch.Tensor):
            ops.add_rows(x, delta=pending)
            pending = None
        if isinstance(pending, CastActivations):
            pending = None
        if pending is not None and not isinstance(pending, PostNormWrite):
            raise TypeError(f"a residual that is mixed with the embedding cannot follow a block that leaves {type(pending).__name__}")
        linear(ctx, self._operand(ctx, x, pending), self.w_x, x)
        return kept


register_part("residual_input", "mix_with_embedding", MixWithEmbedding)
