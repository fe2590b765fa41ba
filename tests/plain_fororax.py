"""A plain, slow implementation of the Fororax design in float64, one function per mechanism.

It shares no code with the engine: it takes a configuration dict (the keys of config.json) and a dict of tensors by
name (numpy arrays), runs one whole sequence, and returns the logits and the residual stream after every layer.
Everything is written from the design's equations:

* the input: a token's row of the table times a constant, plus the position's row of a second table;
* a layer: x = rms(alpha x + mixer(x)) w1; x = rms(alpha x + ff(x)) w2: the stream is what a norm made of the SUM, and
  the parts read the stream itself;
* mixer "attention": grouped heads, a norm per head over q and over k, score = (q . k) scale - r1_h ln(1 + r2_h (i - j)),
  softmax over the keys up to the query; a layer may use an earlier layer's keys and values with its own queries;
* mixer "attention_2": biases on q, k, v and the output, a norm per head over q and over k, no positions, a learned
  number per head in the softmax's denominator; then the heads' weights are mixed, w'_h = sum_g T[h, g] w_g, and head h
  applies w'_h to its own key/value head's values; an element-wise sigmoid gate before the output matrix;
* feed-forward: experts down(g sigmoid(1.702 g) (u + 1)) with g and u cut off at a limit, chosen by softmax scores plus a
  correction, weighted by the scores without it; the last few "experts" hand the input on as it is; one more expert for
  every token, times a sigmoid of one number per token;
* the output: the final norm, the head matrix, cap tanh(. / cap).
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    x = np.asarray(x, dtype=np.float64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * np.asarray(w, dtype=np.float64)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=np.float64)))


def linear(x, tensors, name, bias=False):
    y = x @ np.asarray(tensors[name], dtype=np.float64).T
    return y + np.asarray(tensors[name + ".b"], dtype=np.float64) if bias else y


# ---- the input and the sum a norm is taken of ----------------------------------------------------------------------
def embed(tensors, tokens, positions, scale):
    table, pos = np.asarray(tensors["embed"], dtype=np.float64), np.asarray(tensors["pos"], dtype=np.float64)
    return table[list(tokens)] * scale + pos[list(positions)]


def norm_of_sum(x, y, alpha, w, eps):
    return rms_norm(alpha * x + y, w, eps)


# ---- attention -----------------------------------------------------------------------------------------------------
def log_distance_bias(r1, r2, positions):
    """[H, T, T]: what is taken off the score of (query, key) per head."""
    p = np.asarray(positions, dtype=np.float64)
    d = np.maximum(p[:, None] - p[None, :], 0.0)
    r1, r2 = (np.asarray(r, dtype=np.float64)[:, None, None] for r in (r1, r2))
    return r1 * np.log(1.0 + r2 * d[None])


def causal_weights(scores, positions, sinks=None):
    """scores [H, T, T]: weights over the keys up to each query; ``sinks`` [H]: numbers whose exponentials join the
    denominators."""
    p = np.asarray(positions)
    seen = p[None, :] <= p[:, None]
    s = np.where(seen[None], scores, -np.inf)
    m = s.max(-1)
    if sinks is not None:
        sinks = np.asarray(sinks, dtype=np.float64)[:, None]
        m = np.maximum(m, sinks)
    e = np.exp(s - m[..., None])
    den = e.sum(-1)
    if sinks is not None:
        den = den + np.exp(sinks - m)
    return e / den[..., None]


def mix_heads(weights, talk):
    """weights [H, T, T]: w'_h = sum_g talk[h, g] w_g."""
    return np.einsum("hg,gij->hij", np.asarray(talk, dtype=np.float64), weights)


def attention_rows(q, k, v, scale, positions, r1=None, r2=None, sinks=None, talk=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] of one sequence, norms already taken.  Returns [T, H, V]."""
    q, k, v = (np.asarray(a, dtype=np.float64) for a in (q, k, v))
    H, G = q.shape[1], k.shape[1]
    own = [h // (H // G) for h in range(H)]
    s = np.stack([q[:, h] @ k[:, own[h]].T for h in range(H)]) * scale
    if r1 is not None:
        s = s - log_distance_bias(r1, r2, positions)
    w = causal_weights(s, positions, sinks)
    if talk is not None:
        w = mix_heads(w, talk)
    return np.stack([w[h] @ v[:, own[h]] for h in range(H)], axis=1)


def keys_values(m, tensors, prefix, h, eps, biased):
    """What a layer with projections of its own caches per token: normed keys and values."""
    T, G = h.shape[0], m["kv_heads"]
    k = linear(h, tensors, prefix + "mix.k", biased).reshape(T, G, m["dim"])
    v = linear(h, tensors, prefix + "mix.v", biased).reshape(T, G, m["vdim"])
    return rms_norm(k, tensors[prefix + "mix.k.norm"], eps), v


def attention(m, tensors, prefix, h, positions, k, v, eps):
    T = h.shape[0]
    q = rms_norm(linear(h, tensors, prefix + "mix.q").reshape(T, m["heads"], m["dim"]), tensors[prefix + "mix.q.norm"], eps)
    o = attention_rows(q, k, v, m["scale"], positions, r1=tensors[prefix + "mix.r1"], r2=tensors[prefix + "mix.r2"])
    return linear(o.reshape(T, -1), tensors, prefix + "mix.o")


def attention_2(m, tensors, prefix, h, positions, k, v, eps):
    T = h.shape[0]
    q = linear(h, tensors, prefix + "mix.q", True).reshape(T, m["heads"], m["dim"])
    q = rms_norm(q, tensors[prefix + "mix.q.norm"], eps)
    o = attention_rows(q, k, v, m["scale"], positions, sinks=tensors[prefix + "mix.sink"], talk=tensors[prefix + "mix.talk"])
    o = o.reshape(T, -1) * sigmoid(linear(h, tensors, prefix + "mix.g"))
    return linear(o, tensors, prefix + "mix.o", True)


# ---- feed-forward --------------------------------------------------------------------------------------------------
def gated_product(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(tensors, prefix, h, limit):
    return linear(gated_product(linear(h, tensors, prefix + "gate"), linear(h, tensors, prefix + "up"), limit), tensors,
                  prefix + "down")


def route(h, router, correction, top):
    """Per row: the chosen outputs, their weights, and the gap between the last chosen choice score and the next."""
    z = h @ np.asarray(router, dtype=np.float64).T
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    c = s + np.asarray(correction, dtype=np.float64)
    order = np.argsort(-c, axis=-1, kind="stable")
    ids = order[:, :top]
    ranked = np.take_along_axis(c, order, -1)
    gap = ranked[:, top - 1] - ranked[:, top] if c.shape[1] > top else np.full(len(c), np.inf)
    return ids, np.take_along_axis(s, ids, -1), gap


def routed_ff(f, tensors, prefix, h):
    r = f["router"]
    ids, weights, gap = route(h, tensors[prefix + "router"], tensors[prefix + "correction"], r["top"])
    out = np.zeros_like(h)
    for i in range(r["experts"] + r.get("identity", 0)):
        row, place = np.nonzero(ids == i)
        if len(row) == 0:
            continue
        y = h[row] if i >= r["experts"] else expert(tensors, f"{prefix}e{i}.", h[row], f["expert"]["limit"])
        out[row] += weights[row, place][:, None] * y
    if f.get("shared") is not None:
        out = out + sigmoid(linear(h, tensors, prefix + "shared.sg")) * expert(tensors, prefix + "shared.", h, f["shared"]["limit"])
    return out, gap


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ---- the model -----------------------------------------------------------------------------------------------------
def forward(cfg, tensors, tokens):
    """Logits [T, vocab], the residual stream after every layer [L, T, width], and per routed layer the rows' gaps
    between the last chosen expert's choice score and the first one left out."""
    positions = np.arange(len(tokens))
    eps, alpha = cfg["norm"]["eps"], cfg.get("postln_alpha", 1.0)
    x = embed(tensors, tokens, positions, (cfg.get("embedding") or {}).get("scale", 1.0))
    kept, streams, gaps = {}, [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        src = m.get("kv_from")
        if src is None:
            src = i
            kept[i] = keys_values(m, tensors, p, x, eps, layer["type"] == "attention_2")
        mixer = attention if layer["type"] == "attention" else attention_2
        x = norm_of_sum(x, mixer(m, tensors, p, x, positions, *kept[src], eps), alpha, tensors[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y, gaps[i] = routed_ff(layer["mlp"], tensors, p + "mlp.", x)
            x = norm_of_sum(x, y, alpha, tensors[p + "norm2"], eps)
        streams.append(x.copy())
    logits = linear(rms_norm(x, tensors["final.norm"], eps), tensors, "head")
    if cfg.get("logit_softcap"):
        logits = soft_cap(logits, cfg["logit_softcap"])
    return logits, np.stack(streams), gaps
