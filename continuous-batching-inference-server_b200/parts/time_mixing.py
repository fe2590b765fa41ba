"""Time mixing: a linear recurrence whose decays are made from the token (the RWKV family)."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorDecl
from .base import Delta, Mixer, StateNeed, register_mixer

BLENDS = ("r", "k", "v", "g", "w")


class TimeMixing(Mixer):
    """With h' the row before a token's row (zeros ahead of a sequence), every projection reads its own blend
    h + (h' - h) * mu_s: r, k, v and a gate from matrices ``[heads * dim, width]``, and the decay of every head's key
    channels from a narrow one, w = exp(-exp(W_2 tanh(W_1 blend_w) + w0)).  In 32-bit, per head:

        o = (S + diag(u) k v^T)^T r;   S <- diag(w) S + k v^T          (u: a bonus for the current token alone)

    Each head's o is divided by its root mean square (eps inside the root); the heads side by side are multiplied by a
    weight and by silu of the gate, and projected out.

    Per request the mixer keeps S and the last row h' (zeros at the start), 32-bit; a step walks each segment's rows in
    order from there, so prompt portions cut anywhere, single decoded tokens and whole prompts give the same values.
    Nothing is cached per token.  The blends are one kernel, their products one more for a few rows (``ops.linear_blends``).

    ``rank``: the narrow matrix's rows.  ``names``: what follows the layer's prefix in the names of r, k, v, the gate, the
    decay's two matrices and w0, u, the norm's weight, the output matrix and the stem of the blends' weights."""

    scales_heads = True

    def __init__(self, width: int, heads: int, dim: int, rank: int, eps: float,
                 names=("mix.r", "mix.k", "mix.v", "mix.g", "mix.w1", "mix.w2", "mix.w0", "mix.u", "mix.norm", "mix.o", "mix.mu.")):
        self.width, self.heads, self.dim, self.rank, self.eps = int(width), int(heads), int(dim), int(rank), float(eps)
        if not 0 < self.dim <= ops.TIME_MIXING_MAX_DIM:
            raise ValueError(f"dim={dim} is outside 1..{ops.TIME_MIXING_MAX_DIM}, what the recurrence kernel takes")
        if self.rank < 1:
            raise ValueError(f"rank={rank} must be positive")
        self.d = self.heads * self.dim
        self.heads_width = self.d
        self.factor = 1.0
        self.names = tuple(names)
        # a request's state: S, then the last row, each rounded up to 16 bytes
        self.s_floats = -(-self.d * self.dim // 4) * 4
        self.w_in = self.w_2 = self.w_0 = self.u = self.mu = self.norm_w = self.w_out = None

    def scale_heads(self, factor):
        self.factor = float(factor)

    def state_need(self):
        return StateNeed((self.s_floats + -(-self.width // 4) * 4,), torch.float32)

    def tensors(self, prefix):
        n = [prefix + s for s in self.names]
        W, d = self.width, self.d
        return ([TensorDecl(k, (d, W)) for k in n[:4]]
                + [TensorDecl(n[4], (self.rank, W)), TensorDecl(n[5], (d, self.rank)), TensorDecl(n[6], (d,), "vector"),
                   TensorDecl(n[7], (self.heads, self.dim), "vector"), TensorDecl(n[8], (d,), "norm_weight"), TensorDecl(n[9], (W, d))]
                + [TensorDecl(n[10] + s, (W,), "vector") for s in BLENDS])

    def load(self, prefix, tensors, dtype, device):
        n = [prefix + s for s in self.names]
        self.w_in = torch.cat([self._matrix(tensors[k], dtype, device) for k in n[:5]]).contiguous()     # r | k | v | gate | narrow
        self.w_2 = self._matrix(tensors[n[5]], dtype, device)
        self.w_0 = self._vector(tensors[n[6]], device)
        self.u = self._vector(tensors[n[7]], device).reshape(-1)
        self.norm_w = self._vector(tensors[n[8]], device) * self.factor
        self.w_out = self._matrix(tensors[n[9]], dtype, device)
        self.mu = torch.stack([self._vector(tensors[n[10] + s], device) for s in BLENDS]).contiguous()

    def streamed_weights(self):
        return [self.w_in, self.w_2, self.w_out]

    def forward_heads(self, ctx, h, cache, state, out):
        T, d = h.shape[0], self.d
        blends = torch.empty((T, len(BLENDS) * self.width), dtype=h.dtype, device=h.device)
        ops.token_shift(h, state[:, self.s_floats:], ctx.seg_slot, ctx.row_seq, ctx.cu_rows, self.mu, blends)
        rkvg, narrow = ops.linear_blends(blends, self.w_in, 4, d, "tanh")
        raw = ops.linear(narrow, self.w_2, None, None, out_dtype=torch.float32)          # enters exponentials: 32-bit sums
        y = torch.empty((T, d), dtype=torch.float32, device=h.device)
        ops.time_mixing(rkvg, 0, d, 2 * d, raw, self.w_0, self.u, state, ctx.seg_slot, ctx.cu_rows, ctx.n_segments, self.heads,
                        self.dim, y, max_seg_rows=ctx.max_seg_rows)
        ops.rms_norm(y, self.norm_w, self.eps, out, parts=self.heads, gate=rkvg[:, 3 * d:4 * d], gate_act="silu", gate_after=True)

    def forward(self, ctx, h, cache, state):
        out = torch.empty((h.shape[0], self.d), dtype=h.dtype, device=h.device)
        self.forward_heads(ctx, h, cache, state, out)
        if ops.linear_residual(out, self.w_out, ctx.residual):
            return None
        return Delta(ops.linear(out, self.w_out, None, None, out_dtype=torch.float32))


register_mixer("time_mixing", TimeMixing)
