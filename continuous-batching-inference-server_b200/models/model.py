"""The model: layers put together from registered parts as a ``ModelSpec`` says.

The reference hard-wires one model in ``TransformerRunner::forward_step``
(src/transformer.cpp:65-93): embed, L times (LN, QKV, scatter, attention, O + residual,
LN, FC1, GELU, FC2 + residual), final LN, LM head on all rows.  Here the same order comes
out of the spec's layer list and schedule; the head runs only on the rows whose logits
are wanted.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config import ModelSpec, load_config
from ..kernels import ops
from ..parts import (make_block, make_embedding, make_feed_forward, make_head, make_mixer, make_norm, make_pass_input,
                     make_position)
from ..weights import TensorDecl, check_tensors, read_model_tensors

_DTYPES = {"bfloat16": torch.bfloat16, "bf16": torch.bfloat16, "float32": torch.float32, "fp32": torch.float32,
           torch.bfloat16: torch.bfloat16, torch.float32: torch.float32}


def resolve_dtype(dtype) -> torch.dtype:
    if dtype not in _DTYPES:
        raise ValueError(f"dtype {dtype!r} is not one of bfloat16, float32")
    return _DTYPES[dtype]


class Layer:
    """A block with its parts and the tensor-name prefix of its weights."""

    def __init__(self, spec, index: int, shared: Optional["Layer"] = None):
        """``shared``: the layer whose parts this one runs with (``LayerSpec.weights_from``)."""
        self.spec, self.index, self.shares = spec, index, shared is not None
        if shared is not None:
            for name in ("mixer", "feed_forward", "norm_mixer", "norm_feed_forward", "post_norm_mixer",
                         "post_norm_feed_forward", "side"):
                setattr(self, name, getattr(shared, name))
            self._make_block(spec)
            return
        extra = {"own_kv": False} if spec.cache_source is not None and spec.mixer.kind == "attention" else {}
        self.mixer = make_mixer(spec.mixer, **extra)
        self.feed_forward = make_feed_forward(spec.feed_forward)
        self.norm_mixer = make_norm(spec.norm_mixer)
        self.norm_feed_forward = make_norm(spec.norm_feed_forward)
        self.post_norm_mixer = make_norm(spec.post_norm_mixer) if spec.post_norm_mixer is not None else None
        self.post_norm_feed_forward = (make_norm(spec.post_norm_feed_forward)
                                       if spec.post_norm_feed_forward is not None else None)
        self.side = make_feed_forward(spec.side) if spec.side is not None else None
        self._make_block(spec)

    def _make_block(self, spec):
        extra = {}
        if spec.residual_scale != 1.0 or self.side is not None:
            extra = {"residual_scale": spec.residual_scale, "side": self.side}
        if spec.stream_scale != 1.0:
            extra["stream_scale"] = spec.stream_scale
        self.block = make_block(spec.arrangement, self.mixer, self.feed_forward, self.norm_mixer,
                                self.norm_feed_forward, self.post_norm_mixer, self.post_norm_feed_forward, **extra)
        self.norm_names = tuple(spec.norm_prefixes)
        self.post_norm_names = tuple(spec.post_norm_prefixes)

    def parts(self):
        if self.shares:         # they are listed, loaded and counted with the layer they belong to
            return []
        p = self.spec.prefix
        out = [(p, self.mixer), (p, self.feed_forward), (p + self.norm_names[0], self.norm_mixer),
               (p + self.norm_names[1], self.norm_feed_forward)]
        if self.post_norm_mixer is not None:
            out.append((p + self.post_norm_names[0], self.post_norm_mixer))
        if self.post_norm_feed_forward is not None:
            out.append((p + self.post_norm_names[1], self.post_norm_feed_forward))
        if self.side is not None:
            out.append((p, self.side))
        return out


class Model:
    """Embedding, layers in the order of the schedule, final norm and head: each a part built from its
    ``PartSpec`` through the registries.  This class decides nothing about the architecture."""

    def __init__(self, spec: ModelSpec):
        self.spec = spec
        self.embedding = make_embedding(spec.embedding_spec())
        self.position = make_position(spec.position)
        self.layers: List[Layer] = []
        for i, ls in enumerate(spec.layers):
            src = ls.weights_from
            if src is not None and not (0 <= src < i and not self.layers[src].shares):
                raise ValueError(f"layer {i} runs with the weights of layer {src}, which is no earlier layer with weights of its own")
            self.layers.append(Layer(ls, i, None if src is None else self.layers[src]))
        self.pass_inputs = [make_pass_input(p) for p in spec.pass_inputs]
        for ls in spec.layers:
            if ls.pass_input is not None and not 0 <= ls.pass_input[0] < len(self.pass_inputs):
                raise ValueError(f"layer {ls.prefix!r} names pass input {ls.pass_input[0]}, which does not exist")
        for i in spec.schedule:
            if not 0 <= i < len(self.layers):
                raise ValueError(f"schedule names layer {i}; the model has {len(self.layers)} layers")
        for ls in spec.layers:
            if ls.cache_source is not None and not 0 <= ls.cache_source < len(self.layers):
                raise ValueError(f"layer {ls.prefix!r} reads the cache of layer {ls.cache_source}, which does not exist")
        self.final_norm = make_norm(spec.final_norm)
        self.head_part = make_head(spec.head_spec())
        self.dtype: Optional[torch.dtype] = None
        self.device = None

    @property
    def token_table(self) -> Optional[torch.Tensor]:
        return self.embedding.table

    @property
    def head(self) -> Optional[torch.Tensor]:
        """The head's matrix ``[vocab, width]`` (the token table itself when the head is tied)."""
        return getattr(self.head_part, "weight", None)

    def all_parts(self):
        """(tensor-name prefix, part) of every part of the model, in loading order."""
        out = [("", self.embedding), ("", self.position)] + [("", p) for p in self.pass_inputs]
        for layer in self.layers:
            out += layer.parts()
        return out + [(self.spec.final_norm_prefix, self.final_norm), ("", self.head_part)]

    # ---- weights -------------------------------------------------------
    def declared(self) -> List[TensorDecl]:
        decls = []
        for prefix, part in self.all_parts():
            decls += part.tensors(prefix)
        return decls

    def load(self, tensors: Dict[str, torch.Tensor], dtype, device="cuda", where="weights") -> "Model":
        dtype = resolve_dtype(dtype)
        check_tensors(self.declared(), tensors, self.spec.ignored_tensors, where)
        self.dtype, self.device = dtype, torch.device(device)
        for prefix, part in self.all_parts():
            if part is self.head_part:
                part.tie(self.embedding)
            part.load(prefix, tensors, dtype, device)
        self.register_weight_order()
        return self

    def register_weight_order(self) -> None:
        """The order in which a step reads the big matrices, for prefetching one ahead (bfloat16 on a GPU)."""
        if self.dtype != torch.bfloat16 or self.device.type != "cuda":
            return
        order = []
        for li in self.spec.schedule:
            layer = self.layers[li]
            if layer.spec.pass_input is not None:
                order += self.pass_inputs[layer.spec.pass_input[0]].streamed_weights()
            order += layer.mixer.streamed_weights() + layer.feed_forward.streamed_weights()
            if layer.side is not None:
                order += layer.side.streamed_weights()
        ops.add_weight_order(order + self.head_part.streamed_weights())

    def weight_bytes(self) -> int:
        """Bytes of all weights a step reads (each once; a tied head counts once; of the embedding's and the
        position encoding's tables a step reads single rows, which do not count)."""
        seen, total = set(), 0
        def add(t):
            nonlocal total
            if isinstance(t, torch.Tensor) and t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                total += t.numel() * t.element_size()
        for _, part in self.all_parts():
            if part is self.embedding or part is self.position:
                continue
            for v in (part.step_weights() if hasattr(part, "step_weights") else vars(part).values()):
                add(v)
        return total

    # ---- one step ------------------------------------------------------
    def forward(self, ctx) -> torch.Tensor:
        """Logits (float32 ``[R, vocab]``) at ``ctx.logit_rows`` for the rows of this step."""
        ctx.shared = {}      # what layers hand to later layers within one step
        x = self.embedding.forward(ctx, self.position)
        for p in self.pass_inputs:
            p.begin(ctx, x)
        pending = None
        sched = self.spec.schedule
        i = 0
        while i < len(sched):
            li = sched[i]
            ahead = self.layers[li].spec.pass_input
            if ahead is not None:
                x, pending = self.pass_inputs[ahead[0]].forward(ctx, x, pending, ahead[1])
            block, cache, state = self.layers[li].block, ctx.layer_cache(li), ctx.layer_state(li)
            key = block.run_key(ctx, cache, state)
            if key is None:
                pending = block.forward(ctx, x, pending, cache, state)
                i += 1
                continue
            # a run of consecutive layers whose blocks can go together (for instance one kernel for all of them)
            run = [(block, cache, state)]
            j = i + 1
            while j < len(sched):
                nxt = self.layers[sched[j]].block
                c2, s2 = ctx.layer_cache(sched[j]), ctx.layer_state(sched[j])
                if self.layers[sched[j]].spec.pass_input is not None or type(nxt) is not type(block) or nxt.run_key(ctx, c2, s2) != key:
                    break
                run.append((nxt, c2, s2))
                j += 1
            pending = type(block).forward_run(ctx, [r[0] for r in run], x, pending, [r[1] for r in run], [r[2] for r in run])
            i = j
        return self.head_part.forward(ctx, x, pending, self.final_norm)


def declared_tensors(spec: ModelSpec) -> List[TensorDecl]:
    return Model(spec).declared()


def load_model(folder: str, dtype="bfloat16", device="cuda") -> Model:
    """Model of ``folder`` (config.json chooses the architecture; model.safetensors by tensor name)."""
    config = load_config(folder)
    tensors = read_model_tensors(folder)
    if hasattr(config, "with_shapes"):      # a format may leave a size to a tensor's shape
        config = config.with_shapes({name: tuple(t.shape) for name, t in tensors.items()})
    model = Model(config.model_spec())
    model.config = config
    model.load(tensors, dtype, device, where=f"{folder}/model.safetensors")
    return model
