"""Two mixers side by side."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Delta, Mixer, make_mixer, register_mixer


class SideBySide(Mixer):
    """left_scale * left(h) + right_scale * right(h): two mixers (``PartSpec``s of the mixer registry) that read the same
    rows.  ``names``: what follows the layer's prefix ahead of each one's tensor names.  One of them may keep a cache, one a
    state.

    Both mixers offer the rows that go into their last products (``Mixer.forward_heads``); the rows lie side by side and the
    two products run as ONE, over both matrices side by side.  A constant that a mixer applies to its rows for nothing
    (``scales_heads``) is put there; what is left is one factor on the sum (``Delta.scale``), which the norm that adds the
    result applies."""

    def __init__(self, width: int, left, right, left_scale: float = 1.0, right_scale: float = 1.0,
                 names=("mix.left.", "mix.right.")):
        self.width, self.names = int(width), tuple(names)
        self.left, self.right = make_mixer(left), make_mixer(right)
        for m in (self.left, self.right):
            if not m.heads_width:
                raise ValueError(f"{type(m).__name__} does not offer the rows of its last product: it cannot stand side by side")
        if self.left.cache_need() is not None and self.right.cache_need() is not None:
            raise ValueError("of two mixers side by side only one may keep a cache")
        if self.left.state_need() is not None and self.right.state_need() is not None:
            raise ValueError("of two mixers side by side only one may keep a state")
        ls, rs = float(left_scale), float(right_scale)
        self.keep_left, self.keep_right = ls != 0.0, rs != 0.0      # a mixer times zero still moves its cache and state on
        # scale * (first + ratio * second), the ratio applied by a mixer that can
        if ls == rs or not self.keep_left or not self.keep_right:
            self.scale = ls if self.keep_left else rs
        elif self.right.scales_heads:
            self.right.scale_heads(rs / ls)
            self.scale = ls
        elif self.left.scales_heads:
            self.left.scale_heads(ls / rs)
            self.scale = rs
        else:
            raise ValueError("neither of two mixers with unlike constants can scale its rows")
        self.w_out = None

    def cache_need(self):
        return self.left.cache_need() or self.right.cache_need()

    def state_need(self):
        return self.left.state_need() or self.right.state_need()

    def tensors(self, prefix):
        return self.left.tensors(prefix + self.names[0]) + self.right.tensors(prefix + self.names[1])

    def load(self, prefix, tensors, dtype, device):
        self.left.load(prefix + self.names[0], tensors, dtype, device)
        self.right.load(prefix + self.names[1], tensors, dtype, device)
        halves = [m.w_out if keep else torch.zeros_like(m.w_out)
                  for m, keep in ((self.left, self.keep_left), (self.right, self.keep_right))]
        self.w_out = torch.cat(halves, dim=1).contiguous()
        self.left.w_out = self.right.w_out = None       # held here, side by side

    def streamed_weights(self):
        return ([w for m in (self.left, self.right) for w in m.streamed_weights() if w is not None]) + [self.w_out]

    def step_weights(self):
        """Every tensor a step reads through the two mixers and this part (for counting bytes)."""
        return [v for m in (self, self.left, self.right) for v in vars(m).values() if isinstance(v, torch.Tensor)]

    def forward(self, ctx, h, cache, state):
        T, n = h.shape[0], self.left.heads_width
        rows = torch.empty((T, n + self.right.heads_width), dtype=h.dtype, device=h.device)
        self.left.forward_heads(ctx, h, cache, state, rows[:, :n])
        self.right.forward_heads(ctx, h, cache, state, rows[:, n:])
        if self.scale == 1.0 and ops.linear_residual(rows, self.w_out, ctx.residual):
            return None
        return Delta(ops.linear(rows, self.w_out, None, None, out_dtype=torch.float32), scale=self.scale)


register_mixer("side_by_side", SideBySide)
