"""Small Fororax configurations with random weights, and the plain implementation's logits."""
import copy

import numpy as np
import torch

import plain_fororax
from figotar_helpers import as_numpy, mixed_schedule  # noqa: F401  (the same schedules)
from vekedra_helpers import make_engine, run_cut, tokens_of  # noqa: F401  (the same engine plumbing)


def attn(heads, kv_heads, dim, vdim, scale, kv_from=None, mlp=None, kind="attention"):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": kind, "mixer": m, "mlp": mlp}


def attn2(*args, **kw):
    return attn(*args, kind="attention_2", **kw)


def moe(experts, top, ff, identity=0, limit=1.0, shared=None, shared_limit=0.8):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared:
        f["shared"] = {"ff": shared, "limit": shared_limit}
    return f


def config(width, vocab, layers, alpha=1.5, scale=0.7, cap=12.0, eps=1e-5, positions=320):
    d = {"architecture": "Fororax", "layers": copy.deepcopy(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width,
         "max_positions": positions}
    if alpha is not None:
        d["postln_alpha"] = alpha
    if scale is not None:
        d["embedding"] = {"scale": scale}
    if cap is not None:
        d["logit_softcap"] = cap
    return d


# every mechanism several times: grouped heads, values of another width than keys, keys and values read from an earlier
# layer (once from a layer of the other kind), identity experts, an expert for all with a limit of its own, a layer
# without a feed-forward
MIXED = config(64, 90, [
    attn(4, 2, 16, 24, 0.25, mlp=moe(5, 2, 24, identity=2, shared=40)),
    attn2(6, 3, 24, 16, 0.3, mlp=moe(6, 3, 16, identity=1, limit=0.6)),
    attn(8, 2, 16, 24, 0.3, kv_from=0, mlp=moe(4, 1, 32, identity=3, shared=16)),
    attn2(4, 2, 8, 8, 0.4, mlp=None),
    attn(6, 3, 24, 16, 0.2, kv_from=1, mlp=moe(7, 4, 24, limit=2.0, shared=24, shared_limit=1.7)),
    attn2(2, 1, 32, 40, 0.2, mlp=moe(3, 2, 40, identity=1, shared=32)),
])
# odd sizes and values that models tend to make equal or 1: widths that are no multiples of 8, one key/value head under
# several query heads and as many key/value heads as query heads, one head, every expert chosen, one expert, only identity
# experts beside one, no constants at all
ODD = config(36, 53, [
    attn(3, 1, 12, 20, 0.3, mlp=moe(3, 3, 20)),
    attn2(5, 5, 6, 10, 0.4, mlp=moe(1, 1, 12, identity=2, shared=20)),
    attn(7, 7, 10, 6, 0.35, mlp=None),
    attn2(3, 1, 20, 12, 0.25, mlp=moe(2, 4, 28, identity=2, shared=9)),
    attn(1, 1, 9, 9, 0.3, mlp=moe(4, 1, 11)),
    attn2(1, 1, 14, 7, 0.3, mlp=moe(5, 2, 16, identity=0, shared=16)),
], alpha=None, scale=None, cap=None, eps=1e-4)
# sizes of the tiled kernels: head sizes 64 and 128 (TMA + tcgen05 prompts, tensor-core decoding), 32 and 80, values
# narrower and wider than keys, groups of more than four and more than eight query heads
WIDE = config(128, 200, [
    attn(4, 2, 64, 64, 0.12, mlp=moe(8, 2, 64, identity=2, shared=64)),
    attn2(8, 4, 64, 64, 0.12, mlp=moe(6, 3, 48, identity=1)),
    attn(2, 1, 128, 128, 0.09, mlp=None),
    attn2(4, 2, 128, 128, 0.09, mlp=moe(4, 2, 64, shared=96)),
    attn(10, 2, 80, 48, 0.11, mlp=moe(4, 1, 32, identity=4, shared=32)),
    attn2(12, 1, 32, 104, 0.17, mlp=None),
    attn(6, 2, 64, 64, 0.12, kv_from=0, mlp=moe(8, 2, 64, shared=40)),
    attn2(6, 3, 80, 48, 0.11, mlp=None),
], alpha=2.2, cap=30.0)
# layers as wide as a small real model's: products of hundreds of rows on the TMA + tcgen05 kernels, experts in tiles
REAL = config(512, 1000, [
    attn(8, 2, 64, 64, 0.125, mlp=moe(8, 2, 352, identity=2, limit=4.0, shared=352, shared_limit=3.0)),
    attn2(8, 2, 64, 64, 0.125, mlp=moe(8, 2, 352, identity=1, limit=4.0, shared=352, shared_limit=3.0)),
    attn(4, 2, 64, 64, 0.125, kv_from=0, mlp=moe(8, 2, 352, limit=4.0)),
], alpha=1.8, scale=3.0, cap=25.0)

ONE_LAYER = {
    "attention": config(64, 80, [attn(4, 2, 16, 24, 0.25, mlp=None)]),
    "attention_2": config(64, 80, [attn2(6, 2, 16, 24, 0.2, mlp=None)]),
    "shared_cache": config(64, 80, [attn(4, 2, 16, 24, 0.25, mlp=None), attn(2, 2, 16, 24, 0.3, kv_from=0, mlp=None)]),
    "routed": config(64, 80, [attn(2, 2, 8, 8, 0.3, mlp=moe(6, 2, 24, identity=2, shared=32))]),
}


def unrouted(cfgd):
    """The configuration without its feed-forwards: for comparisons of chosen tokens in bfloat16, where rounding may send
    a token to another expert."""
    out = copy.deepcopy(cfgd)
    for layer in out["layers"]:
        layer["mlp"] = None
    return out


def make_weights(cfgd, seed, std=0.25, tweak=None, dtype="float32"):
    """Random tensors of the configuration, values exact in bfloat16 (both precisions and the plain implementation
    then see the same numbers); ``tweak(tensors)`` may change some before they are rounded.  For bfloat16 the router's
    corrections lie far apart: fewer choices hang on rounding (in 32-bit the choice changes from token to token)."""
    import cbis_b200 as cb
    from cbis_b200.models import Model
    from cbis_b200.weights import InitScheme, random_tensors
    spec = cb.config_from_dict(cfgd).model_spec()
    tensors = random_tensors(Model(spec).declared(), seed, InitScheme(std, 0.3, 0.2, 0.2), torch.float32, draw_on="cpu")
    W = cfgd["width"]
    for name, t in tensors.items():
        if t.dim() == 2 and name not in ("embed", "pos") and not name.endswith(".talk"):
            t.mul_((W / t.shape[1]) ** 0.5)         # keep activations of order one
        if name in ("embed", "pos"):
            t.mul_(3.0)
        if name.endswith(".sink"):
            t.add_(1.5)                             # a sink that takes a visible share of the denominator
        if name.endswith((".r1", ".r2")):
            t.abs_().add_(0.1)                      # a bias that grows with the distance, at every head's own rate
        if name.endswith(".router"):
            t.mul_(3.0)                             # scores apart from one another: few close calls
        if name.endswith(".correction"):
            t.mul_(2.0 if dtype == "float32" else 12.0)      # a correction that changes which experts are chosen
        if name.endswith(".talk"):
            t.mul_(1.5).add_(0.7 * torch.eye(t.shape[0]))
    if tweak is not None:
        tweak(tensors)
    return {k: v.to(torch.bfloat16).float() for k, v in tensors.items()}


def plain_all(cfgd, tensors, tokens):
    """Logits, the stream after every layer, and the first position at which some routed layer's choice hangs on
    less than 0.02 between two choice scores (the length if there is none)."""
    logits, streams, gaps = plain_fororax.forward(cfgd, as_numpy(tensors), list(tokens))
    close = [int(np.nonzero(g < 0.02)[0][0]) for g in gaps.values() if (g < 0.02).any()]
    return torch.from_numpy(logits), torch.from_numpy(streams), min(close, default=len(tokens))


def rounding_moves(cfgd, tensors, tokens):
    """Per row, how far the plain implementation's own logits move when the products' inputs, and the results that go into
    norms, attention and gated products, are rounded to bfloat16: some rows magnify rounding (a head's query is divided
    by its own size, softmax scores compete), in the engine as here."""
    exact = plain_fororax.linear

    def rounded(x):
        return torch.from_numpy(np.ascontiguousarray(x)).to(torch.bfloat16).double().numpy()

    def linear(x, tensors, name, bias=False):
        y = exact(rounded(x), tensors, name, bias)
        return y if name.endswith(("head", "mix.o", "down")) else rounded(y)
    w = as_numpy(tensors)
    ref = plain_fororax.forward(cfgd, w, list(tokens))[0]
    plain_fororax.linear = linear
    try:
        moved = plain_fororax.forward(cfgd, w, list(tokens))[0]
    finally:
        plain_fororax.linear = exact
    return torch.from_numpy(np.abs(moved - ref).max(1))


def plain(cfgd, tensors, tokens):
    return plain_all(cfgd, tensors, tokens)[0]


def assert_close(got, ref, dtype, what="", first_close=None, tol32=2e-4, moves=None):
    """32-bit: every row within ``tol32``.  bfloat16: every row before the sequence's first routing close call
    (``first_close``; None: there is no routing) within 4 % of the largest logit, and the median row of all too: an
    expert that rounding flips moves a few rows, a fault moves most.  ``moves`` (``rounding_moves``): a row may be off by
    three times what rounding does to it in the plain implementation on top of that."""
    err = (got - ref).abs().max(1).values
    assert torch.isfinite(got).all(), what
    if dtype == "float32":
        assert err.max() < tol32, (what, int(err.argmax()), err.max().item())
        return
    tol = 0.04 * max(1.0, ref.abs().max().item())
    if moves is not None:
        err = (err - 3 * moves).clamp(min=0)
    n = len(err) if first_close is None else first_close
    assert n == 0 or err[:n].max() < tol, (what, int(err[:n].argmax()), err[:n].max().item(), n)
    assert err.median() < tol, (what, err.median().item())
