"""Plain Buludra forward pass: whole sequences, no cache, numpy float64.

One function per mechanism, written from the design's equations. Notation: T tokens, x the residual stream
[T, width], W the dictionary of weights by tensor name, p a tensor-name prefix, m a mixer's entry of the
configuration. Linear weights are [out, in] and applied as x @ W.T. No code is shared with the product package.

  rms_unit            x / sqrt(mean(x^2) + eps)
  turn_halves         pairs (i, i + dims/2) of a head's first `dims` dimensions turned by the position's angles
  query_temperature   1 + coef ln(floor((position + 1) / every) + 1)
  softmax_rows        softmax over the visible keys, optionally with one more term of score 0 in the denominator
  grouped_heads       grouped-query attention from finished q, k, v
  normed_attention    q and k normed per head with a gain, no rotation, query temperature
  null_attention      q and k rotated, then brought to unit RMS; the softmax's denominator has a 1 in it
  gated_linear        linear attention whose state decays per key channel, walked token by token
  matrix_memory       the mLSTM's matrix memory with its stabiliser, walked token by token
  side_by_side        the weighted sum of null_attention and matrix_memory on one input
  pick_experts        softmax scores, best groups by their largest, `top` of them
  gated_ff, routed_ff the dense feed-forward; a token's weighted experts plus the gated shared one
  forward             embedding, layers (some with another layer's weights), norm, capped head
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def log_sigmoid(x):
    return -np.logaddexp(0.0, -x)


def silu(x):
    return x * sigmoid(x)


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def turn_halves(x, rot):
    """x [T, heads, d], row t at position t."""
    dims, half = int(rot["dims"]), int(rot["dims"]) // 2
    f = float(rot["base"]) ** (-2.0 * np.arange(half, dtype=np.float64) / dims)
    a = np.arange(x.shape[0], dtype=np.float64)[:, None, None] * f
    c, s = np.cos(a), np.sin(a)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def query_temperature(T, q_temp):
    p = np.arange(T, dtype=np.float64)
    return 1.0 + float(q_temp["coef"]) * np.log(np.floor((p + 1.0) / float(q_temp["every"])) + 1.0)


def softmax_rows(s, null=False):
    """s [T, T]: row i sees columns 0..i. `null`: the denominator holds exp(0) as well."""
    T = s.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf)
    top = s.max(-1, keepdims=True)
    if null:
        top = np.maximum(top, 0.0)
    w = np.exp(s - top)
    return w / (w.sum(-1, keepdims=True) + (np.exp(-top) if null else 0.0))


def grouped_heads(q, k, v, scale, null=False):
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_rows(q[:, h] @ k[:, g].T * scale, null) @ v[:, g]
    return out.reshape(T, -1)


def project_heads(h, W, name, heads):
    return (h @ W[name].T).reshape(h.shape[0], heads, -1)


def normed_attention(h, W, p, m, eps):
    H, G = int(m["heads"]), int(m["kv_heads"])
    q, k, v = project_heads(h, W, p + "q", H), project_heads(h, W, p + "k", G), project_heads(h, W, p + "v", G)
    q, k = rms_unit(q, eps) * W[p + "q.norm"], rms_unit(k, eps) * W[p + "k.norm"]
    if m.get("q_temp"):
        q = q * query_temperature(h.shape[0], m["q_temp"])[:, None, None]
    return grouped_heads(q, k, v, float(m["scale"])) @ W[p + "o"].T


def null_attention(h, W, p, m, eps):
    H, G = int(m["heads"]), int(m["kv_heads"])
    q, k, v = project_heads(h, W, p + "q", H), project_heads(h, W, p + "k", G), project_heads(h, W, p + "v", G)
    q, k = rms_unit(turn_halves(q, m["rot"]), eps), rms_unit(turn_halves(k, m["rot"]), eps)
    return grouped_heads(q, k, v, float(m["scale"]), null=True) @ W[p + "o"].T


def gated_linear_heads(q, k, v, log_a):
    """q, k, log_a [T, H, dim], v [T, H, vd] -> o [T, H, vd]."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = np.exp(log_a[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hd,hdv->hv", q[t], S)
    return o


def gated_linear(h, W, p, m, eps):
    H, dim = int(m["heads"]), int(m["dim"])
    T = h.shape[0]
    q, k, v = (project_heads(h, W, p + n, H) for n in ("q", "k", "v"))
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    log_a = (log_sigmoid(z) / float(m["tau"])).reshape(T, H, dim)
    o = gated_linear_heads(q * dim ** -0.5, k, v, log_a)
    o = (rms_unit(o, eps) * W[p + "norm"]).reshape(T, -1)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def matrix_memory_heads(q, k, v, log_i, log_f):
    """q, k [T, H, dim], v [T, H, vd], log_i, log_f [T, H] -> o [T, H, vd]."""
    T, H, dim = q.shape
    S, n, mx = np.zeros((H, dim, v.shape[2])), np.zeros((H, dim)), np.zeros(H)
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        new = np.maximum(log_f[t] + mx, log_i[t])
        keep, add = np.exp(log_f[t] + mx - new), np.exp(log_i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        mx = new
        den = np.maximum(np.abs((n * q[t]).sum(-1)), np.exp(-mx)) + 1e-6
        o[t] = np.einsum("hd,hdv->hv", q[t], S) / den[:, None]
    return o


def matrix_memory(h, W, p, m, eps):
    H, dim, cap = int(m["heads"]), int(m["dim"]), float(m["gate_cap"])
    T = h.shape[0]
    q, k, v = (project_heads(h, W, p + n, H) for n in ("q", "k", "v"))
    log_i = cap * np.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    log_f = log_sigmoid(cap * np.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    o = rms_unit(matrix_memory_heads(q * dim ** -0.5, k, v, log_i, log_f), eps).reshape(T, -1)
    return (o * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def side_by_side(h, W, p, m, eps):
    return (float(m["left_scale"]) * null_attention(h, W, p + "left.", m["left"], eps)
            + float(m["right_scale"]) * matrix_memory(h, W, p + "right.", m["right"], eps))


def pick_experts(h, W, p, router, margins=None):
    """(experts [T, top], weights [T, top]) in the order of the choice. `margins`, a list, receives per token the
    smallest gap by which a group or an expert made it into the choice, in router logits (inf: nothing left out)."""
    E, top = int(router["experts"]), int(router["top"])
    z = h @ W[p + "router"].T
    s = np.exp(z - z.max(-1, keepdims=True))
    s = s / s.sum(-1, keepdims=True)
    choice = z.copy()                                     # the order of the scores is the order of the logits
    gap = np.full(h.shape[0], np.inf)
    groups = router.get("groups")
    if groups:
        n, keep = int(groups["count"]), int(groups["keep"])
        best_of = choice.reshape(-1, n, E // n).max(-1)
        best = np.argsort(-best_of, axis=-1, kind="stable")[:, :keep]
        if keep < n:
            ordered = -np.sort(-best_of, axis=-1)
            gap = np.minimum(gap, ordered[:, keep - 1] - ordered[:, keep])
        allowed = np.zeros((h.shape[0], n), dtype=bool)
        np.put_along_axis(allowed, best, True, axis=1)
        choice = np.where(np.repeat(allowed, E // n, axis=1), choice, -np.inf)
    picked = np.argsort(-choice, axis=-1, kind="stable")[:, :top]
    if margins is not None:
        if top < E:
            ordered = -np.sort(-choice, axis=-1)
            gap = np.minimum(gap, ordered[:, top - 1] - ordered[:, top])
        margins.append(gap)
    return picked, np.take_along_axis(s, picked, axis=1)


def gated_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def routed_ff(h, W, p, mlp, margins=None):
    picked, weights = pick_experts(h, W, p, mlp["router"], margins)
    out = np.zeros((h.shape[0], W[p + "e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, w in zip(picked[t], weights[t]):
            out[t] += w * gated_ff(h[t:t + 1], W, f"{p}e{int(e)}.")[0]
    if mlp.get("shared"):
        out += sigmoid(h @ W[p + "shared.sg"].T) * gated_ff(h, W, p + "shared.")
    return out


MIXERS = {"attention": normed_attention, "gla": gated_linear, "parallel": side_by_side}


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = int(cfg["layers"][i]["weights_of"])
    return i


def forward(cfg, W, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence from position 0; `layers_out`, a list, receives the stream behind every
    layer, `margins`, a list, every routed feed-forward's per-token gap between chosen and not chosen."""
    eps = float(cfg["norm"]["eps"])
    x = np.asarray(W["embed"], dtype=np.float64)[np.asarray(tokens, dtype=np.int64)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        x = x + MIXERS[L["type"]](rms_unit(x, eps) * W[p + "norm1"], W, p + "mix.", L["mixer"], eps)
        mlp = L.get("mlp")
        if mlp is not None:
            h = rms_unit(x, eps) * W[p + "norm2"]
            x = x + (gated_ff(h, W, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(h, W, p + "mlp.", mlp, margins))
        if layers_out is not None:
            layers_out.append(x.copy())
    z = (rms_unit(x, eps) * W["final.norm"]) @ np.asarray(W["head"], dtype=np.float64).T
    cap = cfg.get("logit_softcap")
    return float(cap) * np.tanh(z / float(cap)) if cap else z
