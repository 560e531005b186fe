"""Small Sagelorn configurations and weights for the tests (numpy generator; values that bfloat16 holds exactly)."""
import json
import os
import zlib

import numpy as np
import torch


def rotation(dims, base, scaling=None):
    """scaling: (factor, low, high, original)."""
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def _masked(m, window):
    if window:
        m["mask"] = {"size": window}
    return m


def attention(heads, kv_heads, dim, vdim, scale, rot, window=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": _masked(m, window)}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, window=None, scaling=None, named_rank=True):
    """named_rank False: the configuration leaves the queries' latent to the tensors."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": rotation(rot_dim, base, scaling)}
    if named_rank:
        m["q_rank"] = q_rank
    return {"type": "latent_attention", "mixer": _masked(m, window)}


def retention(heads, dim, vdim, decay):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def dense(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def moe(layer, ff, experts, top, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return dict(layer, mlp=mlp)


def bare(layer):
    return dict(layer, mlp=None)


def config(width, vocab, layers, bigram=(97, 29, 13), eps=1e-5, logit_scale=0.7):
    return {"architecture": "Sagelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}


# every mixer and feed-forward, several sizes of each; keys borrowed from layer 0 through a wider and a narrower mask than
# its own, and without any; shared experts of the experts' size and of another, and none
_R0 = rotation(12, 500.0, (4.0, 1.0, 4.0, 60))
HYBRID = config(64, 300, [
    dense(attention(4, 2, 16, 24, 0.3, _R0, 40), 48),
    moe(latent(3, 16, 8, 20, 24, 20, 0.25, 300.0, 24), 24, 6, 2, shared=24),
    moe(attention(4, 2, 16, 24, 0.4, _R0, 70, kv_from=0), 32, 5, 3, shared=40),
    bare(retention(3, 24, 16, [0.9, 0.97, 0.995])),
    dense(attention(2, 1, 24, 40, 0.3, rotation(24, 900.0)), 56),
    moe(retention(2, 8, 40, [0.5, 0.99]), 16, 4, 1),
    dense(attention(4, 2, 16, 24, 0.35, _R0, 9, kv_from=0), 40),
    bare(latent(2, 24, 12, 8, 19, 40, 0.2, 1000.0, named_rank=False)),
])
# sizes that are no multiple of 8 or 4, one head, one expert, top = experts, a window of one token, one bucket, multipliers of
# zero and one, constants of 1, decays of one and zero
ODD = config(44, 131, [
    moe(attention(1, 1, 7, 5, 1.0, rotation(2, 20.0), 1), 12, 1, 1, shared=12),
    moe(latent(5, 3, 2, 7, 9, 5, 1.0, 40.0, 13), 10, 7, 7, shared=9),
    moe(attention(5, 1, 10, 9, 0.5, rotation(6, 50.0, (2.0, 1.0, 2.0, 30)), 33), 30, 9, 2, shared=30),
    bare(retention(3, 11, 3, [1.0, 0.0, 0.75])),
    dense(attention(5, 1, 10, 9, 0.6, rotation(6, 50.0, (2.0, 1.0, 2.0, 30)), kv_from=2), 30),
    moe(retention(1, 5, 7, [0.6]), 9, 2, 2),
], bigram=(1, 0, 1), eps=1e-3, logit_scale=1.0)
ONLY_ATTENTION = config(48, 200, [bare(attention(4, 2, 16, 24, 0.4, rotation(8, 1000.0), 20)),
                                  bare(attention(4, 2, 16, 24, 0.3, rotation(8, 1000.0), 55, kv_from=0))], bigram=(200, 3, 5))
ONLY_LATENT = config(48, 200, [bare(latent(4, 16, 8, 24, 32, 24, 0.3, 1000.0, 30))])
ONLY_RETENTION = config(48, 200, [bare(retention(4, 16, 24, [0.9, 0.99, 0.8, 0.999]))])
ONLY_MOE = config(48, 200, [moe(attention(1, 1, 8, 8, 0.3, rotation(8, 100.0), 64), 56, 12, 3, shared=56)])
# attention so sharp that single keys stand out, windows that end at, before and behind page borders
SHARP = config(64, 150, [
    bare(attention(4, 2, 16, 16, 0.5, rotation(8, 2000.0), 64)),
    dense(latent(3, 12, 4, 16, 24, 20, 0.5, 2000.0, 65), 40),
    bare(attention(4, 2, 16, 16, 0.45, rotation(8, 2000.0), 130, kv_from=0)),
    dense(attention(2, 2, 16, 24, 0.5, rotation(16, 5000.0), 127), 48),
    bare(retention(2, 32, 16, [0.999, 0.9])),
], bigram=(1009, 37, 11))
# widths that the tensor-core kernels take, as they are and padded to them; prompts longer than a tile
WIDE = config(128, 257, [
    moe(attention(6, 3, 64, 56, 0.15, rotation(32, 5000.0, (6.0, 1.0, 4.0, 200)), 100), 64, 8, 2, shared=64),
    dense(latent(5, 40, 16, 32, 48, 72, 0.12, 3000.0, 70), 96),
    moe(attention(6, 3, 64, 56, 0.13, rotation(32, 5000.0, (6.0, 1.0, 4.0, 200)), 250, kv_from=0), 72, 5, 1, shared=40),
    bare(retention(2, 64, 64, [0.98, 0.999])),
    dense(attention(3, 1, 128, 128, 0.1, rotation(128, 10000.0), 64), 64),
    bare(attention(2, 1, 100, 56, 0.1, rotation(32, 10000.0))),
    dense(latent(20, 16, 16, 24, 64, 48, 0.15, 3000.0), 64),
    bare(retention(3, 128, 128, [0.97, 0.9, 0.995])),
])
# the large ends
LARGE = config(96, 400, [
    moe(attention(2, 2, 200, 256, 0.07, rotation(100, 10000.0), 90), 200, 72, 4, shared=104),
    dense(latent(3, 40, 56, 72, 136, 200, 0.1, 10000.0, 150), 104),
    moe(retention(2, 256, 160, [0.99, 0.95]), 64, 72, 3, shared=64),
    bare(retention(1, 200, 256, [0.98])),
], bigram=(100003, 2147483647, 999999937))

CONFIGS = {"hybrid": HYBRID, "odd": ODD, "attention": ONLY_ATTENTION, "latent": ONLY_LATENT, "retention": ONLY_RETENTION,
           "moe": ONLY_MOE, "sharp": SHARP, "wide": WIDE, "large": LARGE}
UNNAMED_Q_RANK = 19


def tensor_shapes(cfg, q_rank=UNNAMED_Q_RANK):
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, D), "final.norm": (D,), "head": (V, D)}
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        s[p + "norm1"] = (D,)
        if mlp:
            s[p + "norm2"] = (D,)
            if mlp["kind"] == "dense":
                s.update({p + "mlp.gate": (mlp["ff"], D), p + "mlp.up": (mlp["ff"], D), p + "mlp.down": (D, mlp["ff"])})
            else:
                s[p + "mlp.router"] = (mlp["router"]["experts"], D)
                ffs = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
                for q, F in ffs + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
                    s[f"{p}mlp.{q}.up"], s[f"{p}mlp.{q}.down"] = (F, D), (D, F)
        p += "mix."
        H, vd = m["heads"], m["vdim"]
        s[p + "o"] = (D, H * vd)
        if L["type"] == "attention":
            s.update({p + "q": (H * m["dim"], D), p + "q.norm": (H * m["dim"],), p + "sink": (H,)})
            if m.get("kv_from") is None:
                G = m["kv_heads"]
                s.update({p + "k": (G * m["dim"], D), p + "v": (G * vd, D), p + "k.norm": (G * m["dim"],)})
        elif L["type"] == "latent_attention":
            r, rd, qr = m["kv_rank"], m["rot_dim"], m.get("q_rank", q_rank)
            s.update({p + "dq": (qr, D), p + "dq.norm": (qr,), p + "uq": (H * (m["dim"] + rd), qr), p + "dkv": (r + rd, D),
                      p + "dkv.norm": (r,), p + "uk": (H * m["dim"], r), p + "uv": (H * vd, r), p + "g": (H * vd, D)})
        else:
            s.update({p + "q": (H * m["dim"], D), p + "k": (H * m["dim"], D), p + "v": (H * vd, D), p + "g": (H * vd, D)})
    return s


def make_weights(cfg, seed, kind=""):
    """kind "sharp": large queries and keys (single far keys stand out); "steady": choices that hardly ever hang on a narrow gap
    (for bfloat16 runs, where a narrow gap may fall either way and then moves the rows behind it too), see `_steady`."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        n = lambda std: rng.normal(0, std, shape)
        fan = 1.0 / np.sqrt(shape[-1])
        if name in ("embed", "bigram"):
            w = n(1.0)
        elif last in ("norm1", "norm2") or name == "final.norm":      # stored around zero
            w = n(0.2) - 0.4 * (last != "norm")
        elif last == "norm":
            w = (2.2 if kind == "sharp" and not name.endswith("dkv.norm") else 1.0) * (1.0 + n(0.1))
        elif last == "sink":
            w = n(1.0) + (3.0 if kind == "sharp" else 0.5)
        elif last == "router":
            w = n(fan)
        else:
            w = n(fan)
        W[name] = np.asarray(w)
    if kind == "steady":
        _steady(cfg, W, rng)
    return {name: torch.tensor(w, dtype=torch.float32).to(torch.bfloat16) for name, w in W.items()}


def _steady(cfg, W, rng):
    """The stream's first K columns carry the token's own ranking of K experts (the numbers 0 .. K - 1 in some order; of many experts only the
    first twelve differ from zero): no
    sublayer writes there (gains of zero), and a router's row reads one of them, and a little of everything else."""
    K = max(L["mlp"]["router"]["experts"] for L in cfg["layers"] if L.get("mlp") and L["mlp"]["kind"] == "moe")
    for row in W["embed"]:
        row[:K] = np.maximum(rng.permutation(K) - (K - 12 if K > 12 else 0), 0)
    W["bigram"][:, :K] = 0.0
    for name in W:
        if name.endswith((".norm1", ".norm2")):
            W[name][:K] = -1.0
        if name.endswith(".router"):
            W[name] *= 0.06
            W[name][:, :K] = 0.0
            for e, c in enumerate(rng.permutation(K)[: len(W[name])]):
                W[name][e, c] = 1.0


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
    kind = {"sharp": "sharp", "hybrid": "steady", "wide": "steady", "odd": "steady", "large": "steady"}.get(name, "")
    return make_weights(CONFIGS[name], zlib.crc32(name.encode()) % 1000, kind)      # a seed that stays with the name


def write_models(root, names=None):
    """name -> (folder, config, weights as float64 numpy)."""
    out = {}
    for name, cfg in CONFIGS.items():
        if names is None or name in names:
            W = weights_of(name)
            out[name] = (write_model(os.path.join(str(root), name), cfg, W), cfg, as_numpy(W))
    return out
