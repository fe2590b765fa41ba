"""A plain, slow implementation of the Vipovik design in float64, one function per mechanism.

It shares no code with the engine: it takes a configuration dict (the keys of config.json) and a dict of tensors by
name (numpy arrays), runs one whole sequence, and returns the logits and the residual stream after every layer run.
Everything is written from the design's equations:

* the input: a token's row of the table times a constant; x0 stands for it;
* a loop: the layers start .. stop - 1 run several times with the same weights; ahead of every pass
  x <- W_in [x; x0] + step[pass];
* a layer: x += mixer(rms(x) w1); x += ff(rms(x) w2);
* the mixer is two mixers side by side on the same rows, left_scale * left + right_scale * right:
  - left: grouped heads, rotated q and k (pairs i and i + dims / 2, frequencies slowed down by pair index, cosines and
    sines lengthened), q and k of every head then divided by their root mean square, score = cap tanh(q . k scale / cap),
    softmax over the keys j <= i with i - j < size or j < keep_first;
  - right: the recurrence S <- diag(w_t) S + k_t v_t^T read as o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t, every
    projection reading its own blend of a token's row and the row before it, the decay w_t made from the token's row;
* feed-forward: down gelu(up h) with the erf form, or routed experts whose projections are cut off at a limit, chosen
  and weighted by softmax scores divided by the sum of the chosen ones;
* the output: the final norm, the token table itself.
"""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, w, eps):
    """``w`` None: no weight."""
    x = np.asarray(x, dtype=np.float64)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * np.asarray(w, dtype=np.float64)


def sigmoid(z):
    z = np.asarray(z, dtype=np.float64)
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def gelu(z):
    z = np.asarray(z, dtype=np.float64)
    return 0.5 * z * (1.0 + np.vectorize(math.erf, otypes=[np.float64])(z / math.sqrt(2.0)))


def linear(x, tensors, name):
    return x @ np.asarray(tensors[name], dtype=np.float64).T


# ---- the input and the loop ----------------------------------------------------------------------------------------
def embed(tensors, tokens, scale):
    return np.asarray(tensors["embed"], dtype=np.float64)[list(tokens)] * scale


def pass_input(tensors, x, x0, t):
    """What stands ahead of pass t: W [x; x0] and the pass's own vector."""
    return linear(np.concatenate([x, x0], axis=-1), tensors, "loop.in") + np.asarray(tensors["loop.step"], dtype=np.float64)[t]


def run_order(n_layers, loop):
    """[(layer, number of the pass or None, whether the pass begins here)]."""
    if loop is None:
        return [(i, None, False) for i in range(n_layers)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None, False) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t, i == a) for i in range(a, b)]
    return out + [(i, None, False) for i in range(b, n_layers)]


# ---- left: attention -----------------------------------------------------------------------------------------------
def frequencies(rot):
    """(frequency of every pair, what cosines and sines are multiplied by)."""
    n, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=np.float64)
    s = rot.get("scaling")
    if s is None:
        return f, 1.0
    place = lambda turns: n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(place(s["fast"])), 0), min(math.ceil(place(s["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, H, D]: the first rot dims of every head turned by the position."""
    x = np.array(x, dtype=np.float64)
    if rot is None or not rot["dims"]:
        return x
    f, length = frequencies(rot)
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * f
    c, s, half = np.cos(a) * length, np.sin(a) * length, rot["dims"] // 2
    u, v = x[..., :half].copy(), x[..., half:2 * half].copy()
    x[..., :half], x[..., half:2 * half] = u * c - v * s, v * c + u * s
    return x


def seen(positions, mask):
    """[T, T]: whether the query of row i sees the key of row j."""
    p = np.asarray(positions)
    i, j = p[:, None], p[None, :]
    ok = j <= i
    if mask is not None:
        ok &= (i - j < mask["size"]) | (j < (mask.get("keep_first") or 0))
    return ok


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


def attention_rows(q, k, v, scale, positions, cap, mask):
    """q [T, H, D], k [T, G, D], v [T, G, V] of one sequence, as the scores read them.  Returns [T, H, V]."""
    q, k, v = (np.asarray(a, dtype=np.float64) for a in (q, k, v))
    H, G = q.shape[1], k.shape[1]
    ok, out = seen(positions, mask), []
    for h in range(H):
        g = h // (H // G)
        s = np.where(ok, soft_cap(q[:, h] @ k[:, g].T * scale, cap), -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out.append(e / e.sum(-1, keepdims=True) @ v[:, g])
    return np.stack(out, axis=1)


def attention(m, tensors, prefix, h, positions, eps):
    T = h.shape[0]
    q = linear(h, tensors, prefix + "q").reshape(T, m["heads"], m["dim"])
    k = linear(h, tensors, prefix + "k").reshape(T, m["kv_heads"], m["dim"])
    v = linear(h, tensors, prefix + "v").reshape(T, m["kv_heads"], m.get("vdim") or m["dim"])
    q, k = (rms_norm(rotate(a, positions, m.get("rot")), None, eps) for a in (q, k))
    o = attention_rows(q, k, v, m["scale"], positions, m.get("softcap"), m.get("mask"))
    return linear(o.reshape(T, -1), tensors, prefix + "o")


# ---- right: the recurrence -----------------------------------------------------------------------------------------
def shifted(h, before=None):
    """The row before every row; ``before`` (None: zeros) stands before the first."""
    first = np.zeros((1, h.shape[1])) if before is None else np.asarray(before, dtype=np.float64)[None]
    return np.concatenate([first, h[:-1]])


def blend(h, h_before, mu):
    return h + (h_before - h) * np.asarray(mu, dtype=np.float64)


def decays(mix_w, w1, w2, w0):
    """exp(-exp(w2 tanh(w1 mix_w) + w0)) per channel."""
    w1, w2, w0 = (np.asarray(a, dtype=np.float64) for a in (w1, w2, w0))
    return np.exp(-np.exp(np.tanh(mix_w @ w1.T) @ w2.T + w0))


def recurrence(r, k, v, w, u, state=None):
    """r, k, v, w [T, H, D], u [H, D]; state [H, D, D] (key row, value column), zeros if None.  Returns ([T, H, D], state)."""
    r, k, v, w, u = (np.asarray(a, dtype=np.float64) for a in (r, k, v, w, u))
    T, H, D = r.shape
    S = np.zeros((H, D, D)) if state is None else np.array(state, dtype=np.float64)
    out = np.zeros((T, H, D))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    return out, S


def time_mixing(m, tensors, prefix, h, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    hb = shifted(h)
    mix = {s: blend(h, hb, tensors[prefix + "mu." + s]) for s in "rkvgw"}
    r, k, v = (linear(mix[s], tensors, prefix + s).reshape(T, H, D) for s in "rkv")
    g = linear(mix["g"], tensors, prefix + "g")
    w = decays(mix["w"], tensors[prefix + "w1"], tensors[prefix + "w2"], tensors[prefix + "w0"]).reshape(T, H, D)
    o, _ = recurrence(r, k, v, w, tensors[prefix + "u"])
    o = rms_norm(o, None, eps).reshape(T, -1) * np.asarray(tensors[prefix + "norm"], dtype=np.float64)
    return linear(o * (g * sigmoid(g)), tensors, prefix + "o")


# ---- feed-forward --------------------------------------------------------------------------------------------------
def dense_ff(tensors, prefix, h):
    return linear(gelu(linear(h, tensors, prefix + "up")), tensors, prefix + "down")


def gated_product(g, u, limit):
    if limit:
        g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(tensors, prefix, h, limit):
    return linear(gated_product(linear(h, tensors, prefix + "gate"), linear(h, tensors, prefix + "up"), limit), tensors,
                  prefix + "down")


def route(h, router, top):
    """Per row: the chosen experts, their weights, and the gap between the last chosen score and the next."""
    z = h @ np.asarray(router, dtype=np.float64).T
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    order = np.argsort(-s, axis=-1, kind="stable")
    ranked = np.take_along_axis(s, order, -1)
    gap = ranked[:, top - 1] - ranked[:, top] if s.shape[1] > top else np.full(len(s), np.inf)
    w = ranked[:, :top]
    return order[:, :top], w / (w.sum(-1, keepdims=True) + 1e-20), gap


def routed_ff(f, tensors, prefix, h):
    ids, weights, gap = route(h, tensors[prefix + "router"], f["router"]["top"])
    out = np.zeros_like(h)
    for i in range(f["router"]["experts"]):
        row, place = np.nonzero(ids == i)
        if len(row):
            out[row] += weights[row, place][:, None] * expert(tensors, f"{prefix}e{i}.", h[row], f["expert"].get("limit"))
    return out, gap


# ---- the model -----------------------------------------------------------------------------------------------------
def forward(cfg, tensors, tokens):
    """Logits [T, vocab], the residual stream after every layer run [runs, T, width], and per run of a routed layer the
    rows' gaps between the last chosen expert's score and the first one left out."""
    positions = np.arange(len(tokens))
    eps = cfg["norm"]["eps"]
    x0 = x = embed(tensors, tokens, (cfg.get("embedding") or {}).get("scale", 1.0))
    streams, gaps = [], {}
    for n, (i, t, begins) in enumerate(run_order(len(cfg["layers"]), cfg.get("loop"))):
        layer, p = cfg["layers"][i], f"l{i}."
        m, f = layer["mixer"], layer.get("mlp")
        if begins:
            x = pass_input(tensors, x, x0, t)
        h = rms_norm(x, tensors[p + "norm1"], eps)
        x = (x + m.get("left_scale", 1.0) * attention(m["left"], tensors, p + "mix.left.", h, positions, eps)
             + m.get("right_scale", 1.0) * time_mixing(m["right"], tensors, p + "mix.right.", h, eps))
        if f is not None:
            h = rms_norm(x, tensors[p + "norm2"], eps)
            if f["kind"] == "dense":
                x = x + dense_ff(tensors, p + "mlp.", h)
            else:
                y, gaps[n] = routed_ff(f, tensors, p + "mlp.", h)
                x = x + y
        streams.append(x.copy())
    return linear(rms_norm(x, tensors["final.norm"], eps), tensors, "embed"), np.stack(streams), gaps
