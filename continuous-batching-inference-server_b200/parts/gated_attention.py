"""Attention over the paged cache with separate projections, a distance bias, a query temperature, gates, a norm per head,
sinks and weights mixed across heads."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorDecl
from .base import CacheArray, CacheNeed, Delta, Mixer, register_mixer

NAMES = ("mix.q", "mix.k", "mix.v", "mix.g", "mix.o", "mix.r1", "mix.r2", "mix.sink", "mix.talk")


class GatedAttention(Mixer):
    """q, k, v and a gate come from four matrices stored ``[out, in]`` (q, k, v with biases if ``qkv_bias``), run as
    ONE product.  Keys are ``head_dim`` wide, values ``v_head_dim`` (the two may differ); query head h reads
    key/value head h // (n_head / n_kv_head).  For the query at position p and the key at j <= p:

        score = (q . k) * scale * temperature(p) - bias_h(p - j)
        temperature(p) = 1 + coef * ln(floor((p + 1) / every) + 1)          (``q_temp`` = (coef, every); None: 1)
        bias_h(d) = 2^(-slope_power * (h + 1) / n_head) * d                 (``slope_power`` 0: no such bias)
        bias_h(d) = r1_h * ln(1 + r2_h * d), two learned numbers per head   (``log_bias``)

    inside ``window`` (p - j < window; 0: all keys), ordinary softmax in 32-bit.  The heads side by side are projected out
    (with a bias if ``out_bias``).  No rotation: positions enter through the bias and the temperature only.  Options:

    * ``gate``: "head": head h's output is multiplied by sigmoid(gate_h), one number per token and head read from the
      mixer's input; "element": one number per entry of the heads side by side; None: no gate.  (``head_gate`` True /
      False is the older way to say "head" / None.)
    * ``qk_norm``: every head of q is divided by its own root mean square (``eps`` inside the root) and multiplied by a
      weight as wide as a head, shared by all heads (``<q>.norm``); the same for k, which is cached after it.
    * ``sinks``: a learned number per head whose exponential joins the softmax's denominator (no key, no value).
    * ``talk``: the softmax weights are mixed across heads by a learned matrix T ``[n_head, n_head]`` before they meet the
      values: w'_h = sum_g T[h, g] w_g, head h applies w'_h to its own key/value head's values; sinks are not mixed.
      Decoding rows in bfloat16 mix the weights themselves; elsewhere the attention kernels give every query head's sum
      over the values of EVERY key/value head, and one more kernel takes the sum over g (and the element gate): the order
      of the two sums is exchanged.
    * ``own_kv`` False: the layer has no keys and values of its own (projections, their norm): it reads the pages of the
      layer its cache source names, with its own queries and everything else.

    ``names``: what follows the layer's prefix in the names of q, k, v, the gate, the output matrix, r1, r2, the sinks and
    T; a bias is its matrix's name with ``.b``."""

    def __init__(self, width: int, n_head: int, n_kv_head: int, head_dim: int, v_head_dim: int, scale: float,
                 window: int = 0, qkv_bias: bool = True, slope_power: float = 0.0, q_temp=None, head_gate: bool = True,
                 names=NAMES, gate: str = "default", out_bias: bool = False, log_bias: bool = False, qk_norm: bool = False,
                 eps: float = 1e-5, sinks: bool = False, talk: bool = False, own_kv: bool = True):
        if n_head % n_kv_head:
            raise ValueError(f"n_head={n_head} is not a multiple of n_kv_head={n_kv_head}")
        for what, v in (("head_dim", head_dim), ("v_head_dim", v_head_dim)):
            if not 0 < int(v) <= ops.ATTENTION_MAX_HEAD_DIM:
                raise ValueError(f"{what}={v} is outside 1..{ops.ATTENTION_MAX_HEAD_DIM}, the widest head any "
                                 f"attention kernel takes")
        self.width, self.n_head, self.n_kv_head = int(width), int(n_head), int(n_kv_head)
        self.head_dim, self.v_head_dim = int(head_dim), int(v_head_dim)
        self.scale, self.window, self.own_kv = float(scale), int(window), bool(own_kv)
        self.qkv_bias, self.out_bias = bool(qkv_bias), bool(out_bias)
        self.gate = ("head" if head_gate else None) if gate == "default" else gate
        if self.gate not in ("head", "element", None):
            raise ValueError(f"gate {gate!r} is not one of ['head', 'element', None]")
        self.slope_power, self.log_bias = float(slope_power), bool(log_bias)
        if self.slope_power and self.log_bias:
            raise ValueError("a head has one distance bias: slope_power or log_bias")
        self.q_temp = None if q_temp is None else (float(q_temp[0]), int(q_temp[1]))
        if self.q_temp is not None and self.q_temp[1] < 1:
            raise ValueError(f"q_temp: 'every' must be at least 1, got {self.q_temp[1]}")
        self.qk_norm, self.eps = bool(qk_norm), float(eps)
        self.has_sinks, self.has_talk = bool(sinks), bool(talk)
        if self.has_talk and self.n_head > ops.MIX_HEADS_MAX_HEADS:
            raise ValueError(f"n_head={n_head} is above {ops.MIX_HEADS_MAX_HEADS}, the most heads whose weights are mixed")
        self.d_q, self.d_kv, self.d_v = self.n_head * self.head_dim, self.n_kv_head * self.head_dim, self.n_kv_head * self.v_head_dim
        self.names = tuple(names) + NAMES[len(tuple(names)):]
        self.w_in = self.b_in = self.w_out = self.b_out = None
        self.q_norm_w = self.k_norm_w = self.slopes = self.rates = self.sinks = self.talk = None
        self.sinks_every = None      # with talk: a number per (query head, value head), for kernels that run every such pair

    def cache_need(self):
        if not self.own_kv:
            return None
        return CacheNeed((CacheArray("k", self.n_kv_head, self.head_dim), CacheArray("v", self.n_kv_head, self.v_head_dim)),
                         self.window)

    def _inputs(self):
        """(what follows the prefix in its name, rows, has a bias) of the matrices of the one input product, in column order."""
        n, out = self.names, [(self.names[0], self.d_q, self.qkv_bias)]
        if self.own_kv:
            out += [(n[1], self.d_kv, self.qkv_bias), (n[2], self.d_v, self.qkv_bias)]
        if self.gate is not None:
            out.append((n[3], self.n_head * (self.v_head_dim if self.gate == "element" else 1), False))
        return out

    def tensors(self, prefix):
        n = [prefix + s for s in self.names]
        out = []
        for name, rows, biased in self._inputs():
            out.append(TensorDecl(prefix + name, (rows, self.width)))
            if biased:
                out.append(TensorDecl(prefix + name + ".b", (rows,), "vector"))
        if self.qk_norm:
            out.append(TensorDecl(n[0] + ".norm", (self.head_dim,), "norm_weight"))
            if self.own_kv:
                out.append(TensorDecl(n[1] + ".norm", (self.head_dim,), "norm_weight"))
        if self.log_bias:
            out += [TensorDecl(n[5], (self.n_head,), "vector"), TensorDecl(n[6], (self.n_head,), "vector")]
        if self.has_sinks:
            out.append(TensorDecl(n[7], (self.n_head,), "vector"))
        if self.has_talk:
            out.append(TensorDecl(n[8], (self.n_head, self.n_head), "vector"))
        out.append(TensorDecl(n[4], (self.width, self.n_head * self.v_head_dim)))
        if self.out_bias:
            out.append(TensorDecl(n[4] + ".b", (self.width,), "vector"))
        return out

    def load(self, prefix, tensors, dtype, device):
        n = [prefix + s for s in self.names]
        mats, biases = [], []
        for name, rows, biased in self._inputs():
            mats.append(self._matrix(tensors[prefix + name], dtype, device))
            biases.append(self._vector(tensors[prefix + name + ".b"], device) if biased
                          else torch.zeros(rows, dtype=torch.float32, device=device))
        self.w_in = torch.cat(mats).contiguous()              # q | k | v | gate: one product
        self.b_in = torch.cat(biases).contiguous() if self.qkv_bias else None
        self.w_out = self._matrix(tensors[n[4]], dtype, device)
        self.b_out = self._vector(tensors[n[4] + ".b"], device) if self.out_bias else None
        if self.qk_norm:
            self.q_norm_w = self._vector(tensors[n[0] + ".norm"], device)
            self.k_norm_w = self._vector(tensors[n[1] + ".norm"], device) if self.own_kv else None
        if self.slope_power:
            self.slopes = torch.tensor([2.0 ** (-self.slope_power * (h + 1) / self.n_head) for h in range(self.n_head)],
                                       dtype=torch.float64).to(torch.float32).to(device)
        if self.log_bias:
            self.slopes = self._vector(tensors[n[5]], device)
            self.rates = self._vector(tensors[n[6]], device)
        if self.has_sinks:
            self.sinks = self._vector(tensors[n[7]], device)
        if self.has_talk:
            self.talk = self._vector(tensors[n[8]], device)
            if self.has_sinks:
                self.sinks_every = self.sinks.repeat_interleave(self.n_kv_head).contiguous()

    def streamed_weights(self):
        return [self.w_in, self.w_out]

    def forward(self, ctx, h, cache, state):
        if cache is None:
            raise RuntimeError("attention needs a cache: its own or the layer's it reads")
        T, HV = h.shape[0], self.n_head * self.v_head_dim
        proj = ops.linear(h, self.w_in, self.b_in)
        gate0 = self.d_q + (self.d_kv + self.d_v if self.own_kv else 0)
        if self.qk_norm:
            ops.qk_head_norm(proj, 0, self.n_head, self.d_q, self.n_kv_head if self.own_kv else 0, self.head_dim,
                             self.q_norm_w, self.k_norm_w, self.eps)
        out = torch.empty((T, HV), dtype=h.dtype, device=h.device)
        gate = proj[:, gate0:gate0 + HV] if self.gate == "element" else None
        inside = gate if self.has_talk else None      # the kernels that mix the heads apply the gate too
        ctx.attention(self, proj, cache, ctx.groups[cache.group], out, gate=inside)     # stores k and v (if its own), then attends
        if gate is not None and inside is None:
            ops.gate_mul(gate, out, "sigmoid", out)
        if self.gate == "head":
            ops.head_gate_mul(out, proj[:, gate0:gate0 + self.n_head], self.n_head, out)
        if self.b_out is None and ops.linear_residual(out, self.w_out, ctx.residual):
            return None
        return Delta(ops.linear(out, self.w_out, None, None, out_dtype=torch.float32), self.b_out)


register_mixer("gated_attention", GatedAttention)
