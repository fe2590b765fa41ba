"""What stands ahead of the passes of layers that run several times."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorDecl
from .base import Delta, PassInput, register_pass_input
from .layernorm import NoNorm


class JoinedPassInput(PassInput):
    """x <- W [x; x0] + step_t ahead of pass t: W ``[width, 2 width]``, x first, x0 the embedding's output, step
    ``[passes, width]``.  The two halves of W are products of their own: W_0 x0 is the same ahead of every pass and is taken
    once a step; it is handed on, with the pass's vector, as what the next norm adds to W_x x in its pass over the rows.
    ``names``: the tensor names of W and of the vectors."""

    def __init__(self, width: int, passes: int, names=("loop.in", "loop.step")):
        self.width, self.passes = int(width), int(passes)
        if self.passes < 1:
            raise ValueError(f"passes={passes} must be positive")
        self.names = tuple(names)
        self.as_it_is = NoNorm(self.width)
        self.w_x = self.w_0 = self.steps = None

    def tensors(self, prefix):
        return [TensorDecl(prefix + self.names[0], (self.width, 2 * self.width)),
                TensorDecl(prefix + self.names[1], (self.passes, self.width), "vector")]

    def load(self, prefix, tensors, dtype, device):
        w = self._matrix(tensors[prefix + self.names[0]], dtype, device)
        self.w_x, self.w_0 = w[:, :self.width].contiguous(), w[:, self.width:].contiguous()
        self.steps = self._vector(tensors[prefix + self.names[1]], device)

    def streamed_weights(self):
        return [self.w_x]

    def begin(self, ctx, x):
        rows = self.as_it_is.forward(ctx, x, None)
        ctx.shared[self] = ops.linear(rows, self.w_0, None, None, out_dtype=torch.float32)

    def forward(self, ctx, x, pending, number):
        rows = self.as_it_is.forward(ctx, x, pending)
        return ops.linear(rows, self.w_x, None, None, out_dtype=torch.float32), Delta(ctx.shared[self], self.steps[number])


register_pass_input("joined", JoinedPassInput)
