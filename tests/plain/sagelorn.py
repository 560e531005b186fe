"""Plain Sagelorn forward pass: whole sequences, no cache, numpy float64.

One function per mechanism, written from the design's equations. Notation: T tokens, x the residual stream
[T, width], W the dictionary of weights by tensor name, p a tensor-name prefix, m a mixer's entry of the
configuration. Linear weights are [out, in] and applied as x @ W.T. No code is shared with the product package.

  rms_unit            x / sqrt(mean(x^2) + eps)
  pair_rows           row of the pair table that a token and the one before it name
  pair_frequencies    angular frequency of every rotated pair, with the optional scaling by wavelength
  turn                pairs (i, i + dims/2) or (2i, 2i+1) of a head's first `dims` dimensions turned
  visible             the mask: causal, optionally a window
  softmax_rows        softmax over the visible keys, optionally with one more exponential in the denominator
  own_keys_values     a layer's keys (normed over the whole projection, rotated) and values
  sink_attention      grouped-query attention over given keys and values, with a sink a head
  gated_latent_attention   queries through a latent, keys and values from a latent, elementwise output gate
  retention           linear attention with a fixed decay a head, walked token by token
  gated_ff            the dense feed-forward
  pick_experts        the largest sigmoid scores
  routed_ff           the chosen experts on weighted inputs, plus the shared expert
  forward             embedding with the pair table, layers, norm, scaled head
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def silu(x):
    return x * sigmoid(x)


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def pair_rows(tokens, bigram):
    """tokens of a whole sequence -> rows of the pair table; the sequence's first token has the last row."""
    n, a, b = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    rows = [n]
    for before, now in zip(tokens[:-1], tokens[1:]):
        rows.append((int(before) * a + int(now) * b) % n)
    return np.array(rows, dtype=np.int64)


def pair_frequencies(rot):
    dims, base = int(rot["dims"]), float(rot["base"])
    f = base ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f
    factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for fi in f:
        length = 2.0 * math.pi / fi
        if length < original / high:
            out.append(fi)
        elif length > original / low:
            out.append(fi / factor)
        else:
            s = (original / length - low) / (high - low)
            out.append((1.0 - s) * fi / factor + s * fi)
    return np.array(out)


def turn(x, rot, interleaved):
    """x [T, heads, d], row t at position t."""
    dims = int(rot["dims"])
    a = np.arange(x.shape[0], dtype=np.float64)[:, None, None] * pair_frequencies(rot)
    c, s = np.cos(a), np.sin(a)
    out = x.copy()
    first, second = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., first], x[..., second]
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


def visible(T, mask):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    see = j <= i
    if mask:
        see = see & (i - j < int(mask["size"]))
    return see


def softmax_rows(s, see, extra=None):
    """s [T, T]; `extra`: the denominator holds exp(extra) as well."""
    s = np.where(see, s, -np.inf)
    top = s.max(-1, keepdims=True)
    if extra is not None:
        top = np.maximum(top, extra)
    w = np.exp(s - top)
    return w / (w.sum(-1, keepdims=True) + (np.exp(extra - top) if extra is not None else 0.0))


def own_keys_values(h, W, p, m, eps):
    T, G = h.shape[0], int(m["kv_heads"])
    k = rms_unit(h @ W[p + "k"].T, eps) * W[p + "k.norm"]
    return turn(k.reshape(T, G, -1), m["rot"], False), (h @ W[p + "v"].T).reshape(T, G, -1)


def sink_attention(h, W, p, m, eps, k, v):
    T, H, G = h.shape[0], int(m["heads"]), int(m["kv_heads"])
    q = rms_unit(h @ W[p + "q"].T, eps) * W[p + "q.norm"]
    q = turn(q.reshape(T, H, -1), m["rot"], False)
    see = visible(T, m.get("mask"))
    o = []
    for n in range(H):
        g = n // (H // G)
        o.append(softmax_rows(q[:, n] @ k[:, g].T * float(m["scale"]), see, float(W[p + "sink"][n])) @ v[:, g])
    return np.concatenate(o, axis=-1) @ W[p + "o"].T


def gated_latent_attention(h, W, p, m, eps):
    T, H, dim, rd, r = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["kv_rank"])
    c_q = rms_unit(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (c_q @ W[p + "uq"].T).reshape(T, H, dim + rd)
    d = h @ W[p + "dkv"].T
    c = rms_unit(d[:, :r], eps) * W[p + "dkv.norm"]
    k_r = turn(d[:, None, r:], m["rot"], True)[:, 0]
    q_r = turn(q[..., dim:], m["rot"], True)
    k_u = (c @ W[p + "uk"].T).reshape(T, H, dim)
    v = (c @ W[p + "uv"].T).reshape(T, H, -1)
    see = visible(T, m.get("mask"))
    o = [softmax_rows((q[:, n, :dim] @ k_u[:, n].T + q_r[:, n] @ k_r.T) * float(m["scale"]), see) @ v[:, n] for n in range(H)]
    return (np.concatenate(o, axis=-1) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def retention_heads(q, k, v, decay):
    """q, k [T, H, dim], v [T, H, vd], decay [H] -> o [T, H, vd]."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hd,hdv->hv", q[t], S)
    return o


def retention(h, W, p, m, eps):
    T, H, dim = h.shape[0], int(m["heads"]), int(m["dim"])
    q, k, v = ((h @ W[p + n].T).reshape(T, H, -1) for n in ("q", "k", "v"))
    o = retention_heads(q, k * dim ** -0.5, v, np.array([float(x) for x in m["decay"]]))
    return (rms_unit(o, eps).reshape(T, -1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def gated_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def square_relu_ff(h, W, p):
    u = np.maximum(h @ W[p + "up"].T, 0.0)
    return (u * u) @ W[p + "down"].T


def pick_experts(h, W, p, router, margins=None):
    """(experts [T, top], weights [T, top]) in the order of the choice. `margins`, a list, receives per token the gap
    in router logits between the last expert chosen and the first one left out (inf: none left out)."""
    E, top = int(router["experts"]), int(router["top"])
    z = h @ W[p + "router"].T
    picked = np.argsort(-z, axis=-1, kind="stable")[:, :top]          # the order of the scores is the order of the logits
    if margins is not None:
        ordered = -np.sort(-z, axis=-1)
        margins.append(ordered[:, top - 1] - ordered[:, top] if top < E else np.full(h.shape[0], np.inf))
    return picked, np.take_along_axis(sigmoid(z), picked, axis=1)


def routed_ff(h, W, p, mlp, margins=None):
    picked, weights = pick_experts(h, W, p, mlp["router"], margins)
    out = np.zeros((h.shape[0], W[p + "e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, w in zip(picked[t], weights[t]):
            out[t] += square_relu_ff(w * h[t:t + 1], W, f"{p}e{int(e)}.")[0]
    if mlp.get("shared"):
        out += square_relu_ff(h, W, p + "shared.")
    return out


def forward(cfg, W, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence from position 0; `layers_out`, a list, receives the stream behind every
    layer, `margins`, a list, every routed feed-forward's per-token gap between chosen and not chosen."""
    eps = float(cfg["norm"]["eps"])
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    x = W["embed"][np.asarray(tokens, dtype=np.int64)] + W["bigram"][pair_rows(tokens, cfg["embedding"]["bigram"])]
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        if L["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = own_keys_values(x, W, p + "mix.", m, eps)
            y = sink_attention(x, W, p + "mix.", m, eps, *kept[i if m.get("kv_from") is None else int(m["kv_from"])])
        elif L["type"] == "latent_attention":
            y = gated_latent_attention(x, W, p + "mix.", m, eps)
        else:
            y = retention(x, W, p + "mix.", m, eps)
        x = x + rms_unit(y, eps) * (1.0 + W[p + "norm1"])
        mlp = L.get("mlp")
        if mlp is not None:
            y = gated_ff(x, W, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(x, W, p + "mlp.", mlp, margins)
            x = x + rms_unit(y, eps) * (1.0 + W[p + "norm2"])
        if layers_out is not None:
            layers_out.append(x.copy())
    return (rms_unit(x, eps) * (1.0 + W["final.norm"])) @ W["head"].T * float(cfg["logit_scale"])
