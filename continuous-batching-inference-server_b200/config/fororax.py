"""Typed configuration of Fororax folders.

A Fororax model is a list of unlike layers whose norms stand AFTER the additions: x = norm1(alpha x + mixer(x)),
x = norm2(alpha x + ff(x)), root-mean-square norms with plain weights.  The mixer is attention over grouped heads with a
norm per head over q and k and a bias r1_h ln(1 + r2_h d) by distance ("attention"; a layer may read an earlier layer's
keys and values), or attention without positions with biases, a learned number per head in the softmax's denominator,
weights mixed across heads and an element-wise output gate ("attention_2").  The feed-forward is a routed mixture of
gated ones with cut-off projections, some of whose outputs hand the input on as it is, beside a gated expert for every
token; or absent.  Learned position rows are added to the scaled token rows.  Every size and every constant that may
differ between two models comes from ``config.json``; the tensor names and the gated product's 1.702 and 1 are the
format's.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec
from .vekedra import _get, _int, _num, _only

MIXERS = ("attention", "attention_2")
GATE_BETA, UP_SHIFT = 1.702, 1.0      # of every expert: g * sigmoid(GATE_BETA g) * (u + UP_SHIFT)


def _parse_mixer(kind: str, m: Dict[str, Any], i: int, before) -> Dict[str, Any]:
    where = f"layers[{i}].mixer."
    if kind not in MIXERS:
        raise ConfigError(f"config.json: layers[{i}].type {kind!r} is not one of {sorted(MIXERS)}")
    _only(m, ("dim", "heads", "kv_from", "kv_heads", "scale", "vdim"), where)
    out = {k: _int(m, k, where) for k in ("dim", "heads", "kv_heads")}
    out["vdim"] = _int(m, "vdim", where) if m.get("vdim") is not None else out["dim"]
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}heads={out['heads']} is not a multiple of kv_heads={out['kv_heads']}")
    out["scale"] = _num(m, "scale", where)
    src = m.get("kv_from")
    if src is not None:
        if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
            raise ConfigError(f"config.json: {where}'kv_from' must name an earlier layer, got {src!r}")
        o = before[src].mixer_dict()
        if o.get("kv_from") is not None:
            raise ConfigError(f"config.json: {where}'kv_from'={src}: that layer keeps no keys and values of its own")
        for k in ("kv_heads", "dim", "vdim"):
            if o[k] != out[k]:
                raise ConfigError(f"config.json: {where}{k}={out[k]!r} differs from layer {src}'s {o[k]!r}")
        out["kv_from"] = src
    return out


def _limit(d: Dict[str, Any], where: str) -> float:
    """The cut-off of an expert's projections; 0 stands for none."""
    return _num(d, "limit", where) if d.get("limit") is not None else 0.0


def _parse_mlp(f: Optional[Dict[str, Any]], i: int) -> Optional[Dict[str, Any]]:
    if f is None:
        return None
    where = f"layers[{i}].mlp."
    kind = _get(f, "kind", where)
    if kind != "moe":
        raise ConfigError(f"config.json: {where}'kind' {kind!r} is not one of ['moe']")
    _only(f, ("kind", "expert", "router", "shared"), where)
    expert, router = _get(f, "expert", where), _get(f, "router", where)
    _only(expert, ("ff", "limit"), where + "expert.")
    _only(router, ("experts", "identity", "top"), where + "router.")
    out = {"ff": _int(expert, "ff", where + "expert."), "limit": _limit(expert, where + "expert."),
           "experts": _int(router, "experts", where + "router."), "top": _int(router, "top", where + "router."),
           "identity": _int(router, "identity", where + "router.", 0) if router.get("identity") is not None else 0,
           "shared_ff": 0, "shared_limit": 0.0}
    if out["top"] > out["experts"] + out["identity"]:
        raise ConfigError(f"config.json: {where}router.top={out['top']} exceeds the router's "
                          f"{out['experts'] + out['identity']} outputs")
    shared = f.get("shared")
    if shared is not None:
        _only(shared, ("ff", "limit"), where + "shared.")
        out["shared_ff"], out["shared_limit"] = _int(shared, "ff", where + "shared."), _limit(shared, where + "shared.")
    return out


@dataclass(frozen=True)
class FororaxLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]      # the mixer's sizes and constants, as sorted items
    mlp: Optional[Tuple[Tuple[str, Any], ...]]

    def mixer_dict(self) -> Dict[str, Any]:
        return dict(self.mixer)

    def mlp_dict(self) -> Optional[Dict[str, Any]]:
        return None if self.mlp is None else dict(self.mlp)


@dataclass(frozen=True)
class FororaxConfig:
    vocab: int
    width: int
    norm_eps: float
    max_positions: int
    embedding_scale: float
    postln_alpha: float
    logit_softcap: float            # 0: the logits are not capped
    layers: Tuple[FororaxLayer, ...]
    architecture: str = "Fororax"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "FororaxConfig":
        _only(d, ("architecture", "architectures", "model_type", "embedding", "layers", "logit_softcap", "max_positions",
                  "norm", "postln_alpha", "vocab", "width"), "")
        norm = _get(d, "norm", "")
        _only(norm, ("eps",), "norm.")
        embedding = d.get("embedding") or {}
        _only(embedding, ("scale",), "embedding.")
        raw = _get(d, "layers", "")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw):
            _only(entry, ("type", "mixer", "mlp"), f"layers[{i}].")
            kind = _get(entry, "type", f"layers[{i}].")
            mixer = _parse_mixer(kind, _get(entry, "mixer", f"layers[{i}]."), i, layers)
            mlp = _parse_mlp(entry.get("mlp"), i)
            layers.append(FororaxLayer(kind, tuple(sorted(mixer.items())), None if mlp is None else tuple(sorted(mlp.items()))))

        def optional(src, key, where, default):
            return _num(src, key, where, False) if src.get(key) is not None else default
        return cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), norm_eps=_num(norm, "eps", "norm."),
                   max_positions=_int(d, "max_positions", ""),
                   embedding_scale=optional(embedding, "scale", "embedding.", 1.0),
                   postln_alpha=optional(d, "postln_alpha", "", 1.0),
                   logit_softcap=_num(d, "logit_softcap", "") if d.get("logit_softcap") is not None else 0.0,
                   layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        out = []
        for layer in self.layers:
            f = layer.mlp_dict()
            if f is not None:
                def ffn(ff, limit):
                    return {"ff": ff, "limit": limit} if limit else {"ff": ff}
                g = {"kind": "moe", "expert": ffn(f["ff"], f["limit"]),
                     "router": {"experts": f["experts"], "identity": f["identity"], "top": f["top"]}}
                if f["shared_ff"]:
                    g["shared"] = ffn(f["shared_ff"], f["shared_limit"])
                f = g
            out.append({"type": layer.type, "mixer": layer.mixer_dict(), "mlp": f})
        d = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale}, "layers": out,
             "max_positions": self.max_positions, "norm": {"eps": self.norm_eps}, "postln_alpha": self.postln_alpha,
             "vocab": self.vocab, "width": self.width}
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        return d

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = PartSpec("rmsnorm", {"width": W, "eps": eps, "offset": 0.0, "name": ""})
        none = PartSpec("none", {"width": W})
        specs, ignored = [], []
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer_dict(), layer.mlp_dict()
            source = m.get("kv_from")
            second = layer.type == "attention_2"
            mixer = PartSpec("gated_attention", {
                "width": W, "n_head": m["heads"], "n_kv_head": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
                "scale": m["scale"], "qk_norm": True, "eps": eps, "own_kv": source is None, "qkv_bias": second,
                "out_bias": second, "gate": "element" if second else None, "log_bias": not second, "sinks": second,
                "talk": second})
            if f is None:
                ff = PartSpec("nothing", {"width": W})
                ignored.append(rf"^l{i}\.norm2$")       # a folder may still carry the norm of the part that is absent
            else:
                ff = PartSpec("routed", {"width": W, "inner": f["ff"], "experts": f["experts"], "top": f["top"],
                                         "activation": "silu", "score": "softmax", "renormalize": False, "weight_on": "output",
                                         "correction": True, "identity": f["identity"], "limit": f["limit"],
                                         "beta": GATE_BETA, "up_shift": UP_SHIFT, "shared_inner": f["shared_ff"],
                                         "shared_gate": True, "shared_limit": f["shared_limit"]})
            specs.append(LayerSpec(prefix=f"l{i}.", arrangement="post_norm", mixer=mixer, feed_forward=ff, norm_mixer=norm,
                                   norm_feed_forward=norm if f is not None else none, cache_source=source,
                                   norm_prefixes=("norm1", "norm2"), stream_scale=self.postln_alpha))
        return ModelSpec(width=W, vocab_size=self.vocab, max_positions=self.max_positions,
                         token_embedding=PartSpec("token_table", {"vocab_size": self.vocab, "width": W, "tensor": "embed",
                                                                  "multiplier": self.embedding_scale}),
                         position=PartSpec("learned", {"width": W, "n_positions": self.max_positions, "tensor": "pos"}),
                         layers=tuple(specs), schedule=tuple(range(len(specs))),
                         final_norm=norm, final_norm_prefix="final.norm",
                         head=PartSpec("linear", {"vocab_size": self.vocab, "width": W, "tensor": "head",
                                                  "soft_cap": self.logit_softcap}),
                         ignored_tensors=tuple(ignored))
