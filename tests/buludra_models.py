"""Small Buludra configurations and weights for the tests (numpy generator; values that bfloat16 holds exactly)."""
import json
import os
import zlib

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, scale, q_temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if q_temp:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return {"type": "attention", "mixer": m}


def gla(heads, dim, vdim, tau):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def parallel(left, rot, right, scales):
    """left: (heads, kv_heads, dim, vdim, scale), rot: (dims, base), right: (heads, dim, vdim, gate_cap)."""
    le = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left), rot=dict(zip(("dims", "base"), rot)))
    return {"type": "parallel", "mixer": {"left": le, "right": dict(zip(("heads", "dim", "vdim", "gate_cap"), right)),
                                          "left_scale": scales[0], "right_scale": scales[1]}}


def dense(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def moe(layer, ff, experts, top, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        mlp["shared"] = {"ff": shared}
    return dict(layer, mlp=mlp)


def bare(layer):
    return dict(layer, mlp=None)


def again(layers, j):
    """One more run of layer j's weights."""
    return dict(layers[j], weights_of=j)


def config(width, vocab, layers, eps=1e-5, cap=20.0):
    c = {"architecture": "Buludra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap:
        c["logit_softcap"] = cap
    return c


# every mixer and feed-forward, several sizes of each, layers that run again with another layer's weights
_H = [
    dense(gla(3, 24, 16, 8.0), 48),
    moe(parallel((4, 2, 16, 24, 0.9), (12, 500.0), (2, 8, 16, 6.0), (0.8, 1.3)), 24, 6, 2, groups=(3, 2), shared=40),
    moe(attention(6, 3, 16, 8, 0.4, q_temp=(0.4, 20)), 32, 5, 3, shared=24),
    bare(attention(2, 1, 24, 40, 0.3)),
    dense(parallel((3, 3, 8, 8, 1.2), (8, 90.0), (4, 16, 8, 12.0), (1.5, -0.7)), 56),
]
HYBRID = config(64, 300, _H + [again(_H, 0), again(_H, 1), again(_H, 2), again(_H, 4)])
# sizes that are no multiple of 8 or 4, one head, one expert, top = experts, groups of one expert, constants of 1, no cap
ODD = config(44, 131, [
    moe(gla(1, 5, 7, 1.0), 12, 1, 1, groups=(1, 1)),
    moe(parallel((1, 1, 10, 5, 1.0), (6, 20.0), (3, 6, 5, 1.0), (1.0, 1.0)), 10, 7, 7, groups=(7, 7), shared=9),
    dense(attention(5, 1, 7, 9, 0.5, q_temp=(1.0, 1)), 30),
    moe(attention(3, 3, 6, 11, 1.0, q_temp=(-0.3, 7)), 20, 9, 2, groups=(3, 1), shared=20),
    bare(gla(5, 11, 3, 3.0)),
], eps=1e-3, cap=None)
ONLY_GLA = config(48, 200, [bare(gla(4, 16, 24, 16.0))])
ONLY_PARALLEL = config(48, 200, [bare(parallel((4, 2, 16, 24, 0.5), (16, 1000.0), (2, 16, 32, 10.0), (1.1, 0.6)))])
ONLY_ATTENTION = config(48, 200, [bare(attention(4, 2, 16, 24, 0.4, q_temp=(0.5, 16)))])
ONLY_MOE = config(48, 200, [moe(attention(1, 1, 8, 8, 0.3), 56, 12, 3, groups=(4, 2), shared=32)])
# decays and gates far from their middle: states that vanish within a few tokens, gates at their caps
STRONG = config(64, 150, [bare(gla(2, 32, 24, 0.4)), bare(parallel((2, 1, 16, 16, 0.6), (16, 300.0), (2, 32, 16, 15.0), (0.5, 1.5))),
                          bare(gla(2, 16, 16, 1.0))])
# sharp softmaxes and slow decays: one far token stands out
SHARP = config(64, 150, [
    bare(attention(4, 2, 16, 16, 1.0, q_temp=(0.3, 50))),
    bare(parallel((2, 1, 16, 24, 2.0), (8, 1000.0), (2, 16, 16, 8.0), (1.0, 1.0))),
    bare(gla(2, 16, 16, 32.0)),
])
# heads of the tensor-core kernels' widths (also unequal ones, and ones that are padded to them), states of 128 and 64 x 128
WIDE = config(128, 200, [
    moe(parallel((4, 2, 64, 128, 0.9), (64, 5000.0), (2, 64, 128, 15.0), (1.2, 0.8)), 64, 8, 2, groups=(4, 2), shared=72),
    dense(gla(2, 128, 128, 16.0), 136),
    moe(attention(4, 2, 128, 64, 0.2, q_temp=(0.5, 64)), 48, 6, 2, groups=(2, 1), shared=64),
    bare(attention(6, 2, 40, 72, 0.3)),
    bare(parallel((3, 1, 56, 120, 0.8), (32, 700.0), (3, 40, 56, 9.0), (0.9, 1.1))),
    bare(gla(3, 40, 56, 12.0)),
])
# the large ends: heads of 200 and 256, states of 256 x 160 and 200 x 256, many experts in many groups
LARGE = config(96, 180, [
    bare(gla(1, 256, 160, 16.0)),
    moe(attention(2, 2, 200, 256, 0.07, q_temp=(0.2, 30)), 200, 72, 4, groups=(12, 5), shared=104),
    bare(parallel((2, 1, 256, 40, 0.4), (100, 10000.0), (1, 200, 256, 15.0), (1.0, 0.5))),
])

CONFIGS = {"hybrid": HYBRID, "odd": ODD, "gla": ONLY_GLA, "parallel": ONLY_PARALLEL, "attention": ONLY_ATTENTION, "moe": ONLY_MOE,
           "strong": STRONG, "sharp": SHARP, "wide": WIDE, "large": LARGE}
RANKS = {"odd": 3, "strong": 20, "wide": 16, "large": 40}     # the narrow size of the decay's projection (otherwise 6)


def tensor_shapes(cfg, rank=6):
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        s[p + "norm1"] = (D,)
        mlp = L.get("mlp")
        if mlp:
            s[p + "norm2"] = (D,)
            ffs = ([("mlp.", mlp["ff"])] if mlp["kind"] == "dense" else
                   [(f"mlp.e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])])
            if mlp["kind"] == "moe":
                s[p + "mlp.router"] = (mlp["router"]["experts"], D)
                if mlp.get("shared"):
                    ffs.append(("mlp.shared.", mlp["shared"]["ff"]))
                    s[p + "mlp.shared.sg"] = (1, D)
            for q, F in ffs:
                s[p + q + "gate"] = s[p + q + "up"] = (F, D)
                s[p + q + "down"] = (D, F)
        p += "mix."

        def heads_attention(q, c):
            s.update({q + "q": (c["heads"] * c["dim"], D), q + "k": (c["kv_heads"] * c["dim"], D),
                      q + "v": (c["kv_heads"] * c["vdim"], D), q + "o": (D, c["heads"] * c["vdim"])})

        def memory(q, c):
            H, d, v = c["heads"], c["dim"], c["vdim"]
            s.update({q + "q": (H * d, D), q + "k": (H * d, D), q + "v": (H * v, D), q + "g": (H * v, D), q + "o": (D, H * v)})

        if L["type"] == "attention":
            heads_attention(p, m)
            s[p + "q.norm"] = s[p + "k.norm"] = (m["dim"],)
        elif L["type"] == "gla":
            memory(p, m)
            s.update({p + "norm": (m["vdim"],), p + "a1": (rank, D), p + "a2": (m["heads"] * m["dim"], rank),
                      p + "a2.b": (m["heads"] * m["dim"],)})
        else:
            heads_attention(p + "left.", m["left"])
            r, q = m["right"], p + "right."
            memory(q, r)
            s.update({q + "norm": (r["heads"] * r["vdim"],), q + "i": (r["heads"], D), q + "i.b": (r["heads"],),
                      q + "f": (r["heads"], D), q + "f.b": (r["heads"],)})
    return s


def make_weights(cfg, seed, kind="", rank=6):
    """kind "sharp": large queries, decays near one (single far tokens stand out); "strong": decay and gate inputs of many
    units; "steady": router rows far apart, so that a choice rarely hangs on a narrow gap (for bfloat16 runs, where a narrow
    gap may fall either way)."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        last = name.split(".")[-1]
        n = lambda std: rng.normal(0, std, shape)
        fan = 1.0 / np.sqrt(shape[-1])
        if name == "embed":
            w = n(1.0)
        elif last in ("norm", "norm1", "norm2"):
            w = (2.5 if kind == "sharp" and name.endswith(".q.norm") else 1.0) * (1.0 + n(0.1))
        elif name.endswith("a2.b"):
            w = {"sharp": 6.0, "strong": -1.5}.get(kind, 1.0) + n(3.0 if kind == "strong" else 0.7)
        elif last == "a2":
            w = n((6.0 if kind == "strong" else 1.0) * fan)
        elif name.endswith((".i.b", ".f.b")):
            w = {"sharp": 4.0 if name.endswith(".f.b") else 0.0}.get(kind, 0.5) + n(0.5)
        elif last in ("i", "f"):
            w = n((8.0 if kind == "strong" else 1.0) * fan)
        elif last == "router":
            w = n((6.0 if kind == "steady" else 2.0) * fan)
        elif last in ("g", "sg"):
            w = n(1.5 * fan)
        elif last in ("o", "down"):
            # a recurrence's output is brought to unit size, however small: rows near zero carry rounding at full size, so the
            # sublayers write into the stream at a fraction of its size
            w = n(0.3 * fan)
        else:
            w = n(fan)
        W[name] = torch.tensor(np.asarray(w), dtype=torch.float32).to(torch.bfloat16)
    return W


def as_numpy(W):
    return {n: t.to(torch.float64).numpy() for n, t in W.items()}


def write_model(folder, cfg, W):
    from mynah_slm_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), W)
    return folder


def weights_of(name):
    kind = {"sharp": "sharp", "strong": "strong", "hybrid": "steady", "wide": "steady", "large": "steady"}.get(name, "")
    return make_weights(CONFIGS[name], zlib.crc32(name.encode()) % 1000, kind, RANKS.get(name, 6))      # a seed that stays with the name


def write_models(root, names=None):
    """name -> (folder, config, weights as float64 numpy)."""
    out = {}
    for name, cfg in CONFIGS.items():
        if names is None or name in names:
            W = weights_of(name)
            out[name] = (write_model(os.path.join(str(root), name), cfg, W), cfg, as_numpy(W))
    return out
