"""Small Vipovik configurations with random weights, and the plain implementation's logits."""
import copy

import numpy as np
import torch

import plain_vipovik
from figotar_helpers import as_numpy, mixed_schedule  # noqa: F401  (the same schedules)
from fororax_helpers import assert_close  # noqa: F401  (the same measure)
from vekedra_helpers import make_engine, run_cut, tokens_of  # noqa: F401  (the same engine plumbing)


def left(heads, kv_heads, dim, vdim, scale, window=None, keep=0, cap=None, rot=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    if cap is not None:
        m["softcap"] = cap
    if rot is not None:
        m["rot"] = rot
    return m


def rotation(dims, base=500.0, scaling=(3.0, 60, 12.0, 0.7)):
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def layer(lft, heads, dim, rank, mlp=None, ls=0.8, rs=1.3):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": lft, "right": {"heads": heads, "dim": dim, "decay_rank": rank}, "left_scale": ls, "right_scale": rs}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.2):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit} if limit else {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, loop=None, scale=1.5, eps=1e-5):
    d = {"architecture": "Vipovik", "layers": copy.deepcopy(layers), "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if scale is not None:
        d["embedding"] = {"scale": scale}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# every mechanism several times: grouped heads, values of another width than keys, windows that keep first tokens and that do
# not, no window, rotations of part of a head with and without slowed frequencies, three passes over layers in the middle
MIXED = config(64, 90, [
    layer(left(4, 2, 16, 24, 0.4, 21, 5, 3.0, rotation(12)), 3, 20, 10, dense(72)),
    layer(left(6, 2, 24, 16, 0.3, 13, 9, None, rotation(24)), 4, 16, 24, moe(5, 2, 24), 1.1, 1.1),
    layer(left(2, 2, 16, 16, 0.5, None, 0, 2.0, rotation(16, 90.0, None)), 2, 24, 8, None, -0.7, 0.6),
    layer(left(4, 1, 32, 8, 0.2, 40, 0, 5.0, None), 5, 8, 12, moe(6, 3, 16, 0.7), 1.0, 1.0),
    layer(left(3, 3, 8, 40, 0.5, 6, 33, 1.5, rotation(6, 30.0)), 1, 32, 16, dense(40)),
], loop=(1, 4, 3))
# odd sizes: widths that are no multiples of 4 or 8, windows of one token, first tokens that outnumber the window, every
# expert chosen, one expert, one pass, the loop over the first layer alone, no constants
ODD = config(36, 53, [
    layer(left(3, 1, 12, 20, 0.4, 1, 3, 2.5, rotation(6)), 2, 9, 5, moe(3, 3, 20)),
    layer(left(5, 5, 6, 10, 0.5, 30, 1, None, rotation(2, 20.0)), 3, 7, 3, moe(1, 1, 12, None), 0.5, -0.9),
    layer(left(7, 7, 10, 6, 0.35, 11, 60, 1.1, None), 1, 13, 1, None, 1.4, 0.0),
    layer(left(1, 1, 9, 9, 0.5, None, 0, None, rotation(8, 300.0)), 4, 5, 30, dense(33), 0.0, 1.2),
], loop=(0, 1, 1), scale=None, eps=1e-4)
# sizes of the tiled kernels: head sizes 64 and 128 (TMA + tcgen05 prompts, tensor-core decoding), 80, 96 and 32, windows
# that pass over several key tiles with kept tokens in tiles of their own, recurrences of 64, 96, 128 and 160 channels
WIDE = config(128, 200, [
    layer(left(4, 2, 64, 64, 0.12, 50, 70, 4.0, rotation(64, 9000.0, (4.0, 128, 16.0, 1.0))), 2, 64, 24, dense(96)),
    layer(left(2, 1, 128, 128, 0.09, 90, 3, 30.0, rotation(96)), 1, 128, 16, moe(8, 2, 64)),
    layer(left(10, 2, 80, 48, 0.11, 33, 64, 2.0, rotation(80)), 2, 96, 48, None),
    layer(left(6, 2, 64, 64, 0.12, None, 0, 1.2, rotation(32)), 4, 32, 32, moe(4, 1, 32)),
    layer(left(3, 1, 32, 104, 0.2, 17, 20, None, rotation(32)), 1, 160, 8, dense(64)),
], loop=(0, 2, 2))
# layers as wide as a small real model's: products of hundreds of rows on the TMA + tcgen05 kernels, experts in tiles
REAL = config(512, 1000, [
    layer(left(8, 2, 64, 64, 0.12, 96, 12, 20.0, rotation(64, 10000.0, (4.0, 256, 32.0, 1.0))), 8, 64, 64, dense(1024), 1.0, 0.6),
    layer(left(8, 4, 64, 64, 0.12, 160, 30, 20.0, rotation(64, 10000.0, (4.0, 256, 32.0, 1.0))), 8, 64, 64, moe(8, 2, 352, 4.0), 0.9, 0.9),
], loop=(0, 2, 2), scale=3.0)

_ROT = rotation(16, 100.0)
ONE_LAYER = {
    "attention": config(64, 80, [layer(left(4, 2, 16, 24, 0.4, 19, 6, 3.0, _ROT), 1, 8, 4, None, 1.0, 0.0)]),
    "time_mixing": config(64, 80, [layer(left(1, 1, 8, 8, 0.4), 4, 16, 12, None, 0.0, 1.0)]),
    "side_by_side": config(64, 80, [layer(left(4, 2, 16, 24, 0.4, 19, 6, 3.0, _ROT), 4, 16, 12, None, 1.7, 0.4)]),
    "loop": config(64, 80, [layer(left(4, 2, 16, 16, 0.4, 19, 6, 3.0, _ROT), 2, 16, 12, dense(48))], loop=(0, 1, 4)),
    "routed": config(64, 80, [layer(left(2, 2, 8, 8, 0.4), 2, 8, 4, moe(6, 2, 24))]),
}


def unrouted(cfgd):
    """The configuration with dense feed-forwards for the routed ones: for comparisons of chosen tokens in bfloat16, where
    rounding may send a token to another expert."""
    out = copy.deepcopy(cfgd)
    for l in out["layers"]:
        if l["mlp"] is not None and l["mlp"]["kind"] == "moe":
            l["mlp"] = dense(l["mlp"]["expert"]["ff"])
    return out


def make_weights(cfgd, seed, std=0.25, tweak=None):
    """Random tensors of the configuration, values exact in bfloat16 (both precisions and the plain implementation
    then see the same numbers); ``tweak(tensors)`` may change some before they are rounded."""
    import cbis_b200 as cb
    from cbis_b200.models import Model
    from cbis_b200.weights import InitScheme, random_tensors
    spec = cb.config_from_dict(cfgd).model_spec()
    tensors = random_tensors(Model(spec).declared(), seed, InitScheme(std, 0.3, 0.2, 0.2), torch.float32, draw_on="cpu")
    W = cfgd["width"]
    for name, t in tensors.items():
        if t.dim() == 2 and name != "embed" and not name.endswith((".u", "loop.step")):
            t.mul_((W / t.shape[1]) ** 0.5)         # keep activations of order one
        if name == "loop.in":
            t.mul_(0.3)
        if name == "embed":
            t.mul_(3.0)
        if ".mu." in name:
            t.add_(0.5)                             # blends of every kind, beyond both ends too
        if name.endswith(".w0"):
            t.mul_(5.0).sub_(2.0)                   # decays from a few tokens to hundreds
        if name.endswith(".router"):
            t.mul_(3.0)                             # scores apart from one another: few close calls
    for name in [n for n in tensors if n.endswith("right.u")]:
        # keys that resemble the receptances, positive bonuses: a head's result is divided by its own size, and one that
        # happens to be near zero (at the first token: r . (u k) near zero) would turn with rounding
        stem = name[:-1]
        tensors[name].mul_(3.0).abs_().add_(0.3)
        tensors[stem + "k"] = 0.85 * tensors[stem + "r"] + 0.5 * tensors[stem + "k"]
        tensors[stem + "mu.k"] = tensors[stem + "mu.r"] + 0.3 * (tensors[stem + "mu.k"] - tensors[stem + "mu.r"])
    if tweak is not None:
        tweak(tensors)
    return {k: v.to(torch.bfloat16).float() for k, v in tensors.items()}


def plain_all(cfgd, tensors, tokens):
    """Logits, the stream after every layer run, and the first position at which some routed layer's choice hangs on less
    than 0.02 between two scores (the length if there is none)."""
    logits, streams, gaps = plain_vipovik.forward(cfgd, as_numpy(tensors), list(tokens))
    close = [int(np.nonzero(g < 0.02)[0][0]) for g in gaps.values() if (g < 0.02).any()]
    return torch.from_numpy(logits), torch.from_numpy(streams), min(close, default=len(tokens))


def plain(cfgd, tensors, tokens):
    return plain_all(cfgd, tensors, tokens)[0]


def rounding_moves(cfgd, tensors, tokens):
    """Per row, how far the plain implementation's own logits move when the products' inputs, and the results that go into
    norms, attention, the recurrence and gated products, are rounded to bfloat16."""
    exact = plain_vipovik.linear

    def rounded(x):
        return torch.from_numpy(np.ascontiguousarray(x)).to(torch.bfloat16).double().numpy()

    def linear(x, tensors, name):
        y = exact(rounded(x), tensors, name)
        return y if name.endswith(("embed", ".o", "down", "loop.in")) else rounded(y)
    w = as_numpy(tensors)
    ref = plain_vipovik.forward(cfgd, w, list(tokens))[0]
    plain_vipovik.linear = linear
    try:
        moved = plain_vipovik.forward(cfgd, w, list(tokens))[0]
    finally:
        plain_vipovik.linear = exact
    return torch.from_numpy(np.abs(moved - ref).max(1))
