"""Typed configuration of Vipovik folders.

A Vipovik model is a list of unlike pre-norm layers with root-mean-square norms (plain weights), some of which run several
times in a row with the same weights; ahead of every pass the stream is joined with the embedding's output by one product
and the pass's own vector is added.  A layer's mixer is two mixers side by side on the same rows ("parallel"): attention
over grouped heads, rotated with slowed frequencies, a norm per head after the rotation, a cap on the scores and a sliding
window that keeps the first tokens; and time mixing with decays made from the token.  The feed-forward is down gelu(up h), a
routed mixture of gated ones with cut-off projections, or absent.  The head is the token table.  Every size and every
constant that may differ between two models comes from ``config.json``, but for the rows of the decays' narrow matrix, which
the folder's tensors tell (``with_shapes``) unless ``right.decay_rank`` does; the tensor names and the gated product's 1.702
and 1 are the format's.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .divitar import _freeze, _rot, _thaw
from .fororax import GATE_BETA, UP_SHIFT, _limit
from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec
from .vekedra import _get, _int, _num, _only


def _optional(d: Dict[str, Any], key: str, where: str, default: float) -> float:
    return _num(d, key, where, False) if d.get(key) is not None else default


def _parse_left(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    _only(m, ("dim", "heads", "kv_heads", "mask", "rot", "scale", "softcap", "vdim"), where)
    out = {k: _int(m, k, where) for k in ("dim", "heads", "kv_heads")}
    out["vdim"] = _int(m, "vdim", where) if m.get("vdim") is not None else out["dim"]
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}heads={out['heads']} is not a multiple of kv_heads={out['kv_heads']}")
    out["scale"] = _num(m, "scale", where)
    out["softcap"] = _num(m, "softcap", where) if m.get("softcap") is not None else 0.0
    out["rot"] = _rot(m, where, out["dim"], ("factor", "original", "fast", "slow"))
    mask = m.get("mask")
    out["window"] = out["keep_first"] = 0
    if mask is not None:
        _only(mask, ("keep_first", "size"), where + "mask.")
        out["window"] = _int(mask, "size", where + "mask.")
        out["keep_first"] = _int(mask, "keep_first", where + "mask.", 0) if mask.get("keep_first") is not None else 0
    return out


def _parse_mixer(kind: str, m: Dict[str, Any], i: int) -> Dict[str, Any]:
    if kind != "parallel":
        raise ConfigError(f"config.json: layers[{i}].type {kind!r} is not one of ['parallel']")
    where = f"layers[{i}].mixer."
    _only(m, ("left", "left_scale", "right", "right_scale"), where)
    right = _get(m, "right", where)
    _only(right, ("decay_rank", "dim", "heads"), where + "right.")
    return {"left": _parse_left(_get(m, "left", where), where + "left."),
            "right": {"dim": _int(right, "dim", where + "right."), "heads": _int(right, "heads", where + "right."),
                      "decay_rank": _int(right, "decay_rank", where + "right.") if right.get("decay_rank") is not None else 0},
            "left_scale": _optional(m, "left_scale", where, 1.0), "right_scale": _optional(m, "right_scale", where, 1.0)}


def _parse_mlp(f: Optional[Dict[str, Any]], i: int) -> Optional[Dict[str, Any]]:
    if f is None:
        return None
    where = f"layers[{i}].mlp."
    kind = _get(f, "kind", where)
    if kind == "dense":
        _only(f, ("kind", "ff"), where)
        return {"kind": "dense", "ff": _int(f, "ff", where)}
    if kind == "moe":
        _only(f, ("kind", "expert", "router"), where)
        expert, router = _get(f, "expert", where), _get(f, "router", where)
        _only(expert, ("ff", "limit"), where + "expert.")
        _only(router, ("experts", "top"), where + "router.")
        out = {"kind": "moe", "ff": _int(expert, "ff", where + "expert."), "limit": _limit(expert, where + "expert."),
               "experts": _int(router, "experts", where + "router."), "top": _int(router, "top", where + "router.")}
        if out["top"] > out["experts"]:
            raise ConfigError(f"config.json: {where}router.top={out['top']} exceeds experts={out['experts']}")
        return out
    raise ConfigError(f"config.json: {where}'kind' {kind!r} is not one of ['dense', 'moe']")


@dataclass(frozen=True)
class VipovikLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]      # the mixer's sizes and constants, as sorted items (nested ones too)
    mlp: Optional[Tuple[Tuple[str, Any], ...]]

    def mixer_dict(self) -> Dict[str, Any]:
        return {k: _thaw(v) for k, v in self.mixer}

    def mlp_dict(self) -> Optional[Dict[str, Any]]:
        return None if self.mlp is None else dict(self.mlp)


@dataclass(frozen=True)
class VipovikConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[VipovikLayer, ...]
    loop: Optional[Tuple[int, int, int]] = None     # (first layer, the one after the last, passes); None: every layer runs once
    architecture: str = "Vipovik"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "VipovikConfig":
        _only(d, ("architecture", "architectures", "model_type", "embedding", "layers", "loop", "norm", "vocab", "width"), "")
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
            mixer = _parse_mixer(_get(entry, "type", f"layers[{i}]."), _get(entry, "mixer", f"layers[{i}]."), i)
            mlp = _parse_mlp(entry.get("mlp"), i)
            layers.append(VipovikLayer(entry["type"], _freeze(mixer), None if mlp is None else tuple(sorted(mlp.items()))))
        loop = d.get("loop")
        if loop is not None:
            _only(loop, ("start", "stop", "times"), "loop.")
            loop = (_int(loop, "start", "loop.", 0), _int(loop, "stop", "loop."), _int(loop, "times", "loop."))
            if not loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop.start={loop[0]} and loop.stop={loop[1]} name no run of the "
                                  f"{len(layers)} layers")
        return cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), norm_eps=_num(norm, "eps", "norm."),
                   embedding_scale=_optional(embedding, "scale", "embedding.", 1.0), layers=tuple(layers), loop=loop)

    def to_dict(self) -> Dict[str, Any]:
        out = []
        for layer in self.layers:
            m, f = layer.mixer_dict(), layer.mlp_dict()
            left, right = m["left"], m["right"]
            window, keep = left.pop("window"), left.pop("keep_first")
            if window:
                left["mask"] = {"keep_first": keep, "size": window}
            for key in ("rot", "softcap"):
                if not left[key]:
                    del left[key]
            if not right["decay_rank"]:
                del right["decay_rank"]
            if f is not None and f["kind"] == "moe":
                f = {"kind": "moe", "expert": {"ff": f["ff"], "limit": f["limit"]} if f["limit"] else {"ff": f["ff"]},
                     "router": {"experts": f["experts"], "top": f["top"]}}
            out.append({"type": layer.type, "mixer": m, "mlp": f})
        d = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale}, "layers": out,
             "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d

    def with_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "VipovikConfig":
        """The configuration with the sizes that only a folder's tensors tell."""
        layers = []
        for i, layer in enumerate(self.layers):
            m = layer.mixer_dict()
            shape = shapes.get(f"l{i}.mix.right.w1")
            if not m["right"]["decay_rank"] and shape is not None and len(shape) == 2:
                m["right"]["decay_rank"] = int(shape[0])
                layer = dataclasses.replace(layer, mixer=_freeze(m))
            layers.append(layer)
        return dataclasses.replace(self, layers=tuple(layers))

    def model_spec(self) -> ModelSpec:
        W, eps = self.width, self.norm_eps
        norm = PartSpec("rmsnorm", {"width": W, "eps": eps, "offset": 0.0, "name": ""})
        none = PartSpec("none", {"width": W})
        own, ignored = [], []
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer_dict(), layer.mlp_dict()
            a, b, rot = m["left"], m["right"], m["left"]["rot"]
            if not b["decay_rank"]:
                raise ConfigError(f"layers[{i}].mixer.right.decay_rank: neither config.json nor a tensor l{i}.mix.right.w1 tells it")
            sc = (rot or {}).get("scaling")
            left = PartSpec("rotary_attention", {
                "width": W, "n_head": a["heads"], "n_kv_head": a["kv_heads"], "head_dim": a["dim"], "v_head_dim": a["vdim"],
                "scale": a["scale"], "window": a["window"], "keep_first": a["keep_first"], "cap": a["softcap"],
                "turned_norm": True, "eps": eps, "rot_base": rot["base"] if rot else 10000.0, "rot_dims": rot["dims"] if rot else 0,
                "rot_blend": None if sc is None else (sc["factor"], sc["original"], sc["fast"], sc["slow"]),
                "names": ("q", "k", "v", "o")})
            right = PartSpec("time_mixing", {
                "width": W, "heads": b["heads"], "dim": b["dim"], "rank": b["decay_rank"], "eps": eps,
                "names": ("r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o", "mu.")})
            mixer = PartSpec("side_by_side", {"width": W, "left": left, "right": right, "left_scale": m["left_scale"],
                                              "right_scale": m["right_scale"], "names": ("mix.left.", "mix.right.")})
            if f is None:
                ff = PartSpec("nothing", {"width": W})
                ignored.append(rf"^l{i}\.norm2$")       # a folder may still carry the norm of the part that is absent
            elif f["kind"] == "dense":
                ff = PartSpec("dense", {"width": W, "inner": f["ff"], "activation": "gelu_erf", "names": ("mlp.up", "mlp.down"),
                                        "plain": True})
            else:
                ff = PartSpec("routed", {"width": W, "inner": f["ff"], "experts": f["experts"], "top": f["top"],
                                         "activation": "silu", "score": "softmax", "renormalize": True, "renorm_eps": 1e-20,
                                         "weight_on": "output", "limit": f["limit"], "beta": GATE_BETA, "up_shift": UP_SHIFT})
            own.append(LayerSpec(prefix=f"l{i}.", arrangement="pre_norm_scaled", mixer=mixer, feed_forward=ff, norm_mixer=norm,
                                 norm_feed_forward=norm if f is not None else none, norm_prefixes=("norm1", "norm2")))
        specs, inputs = own, ()
        if self.loop is not None:
            # every pass has caches and states of its own: the later passes are layers that run with the first pass's weights
            start, stop, times = self.loop
            inputs = (PartSpec("joined", {"width": W, "passes": times, "names": ("loop.in", "loop.step")}),)
            specs = list(own[:start])
            for t in range(times):
                for i in range(start, stop):
                    specs.append(dataclasses.replace(own[i], weights_from=i if t else None,
                                                     pass_input=(0, t) if i == start else None))
            specs += own[stop:]
        return ModelSpec(width=W, vocab_size=self.vocab, max_positions=0,      # 0: the design sets no limit; the engine's holds
                         token_embedding=PartSpec("token_table", {"vocab_size": self.vocab, "width": W, "tensor": "embed",
                                                                  "multiplier": self.embedding_scale}),
                         position=PartSpec("none", {"width": W}), layers=tuple(specs), schedule=tuple(range(len(specs))),
                         final_norm=norm, final_norm_prefix="final.norm",
                         head=PartSpec("linear", {"vocab_size": self.vocab, "width": W, "tensor": None}),
                         pass_inputs=inputs, ignored_tensors=tuple(ignored))
