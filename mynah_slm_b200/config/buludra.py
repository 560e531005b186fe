"""Typed configuration of the Buludra design, read from its config.json.

A small decoder-only model whose layers are listed one by one: `layers[i]`
names the layer's mixer (`type`), the mixer's sizes (`mixer`) and its
feed-forward (`mlp`, or null for none). A layer that names another one
(`weights_of`) has no tensors of its own: it runs the other layer's mixer,
feed-forward and norms, with a cache and state of its own. Every size and
every constant that can differ between two models of the design is read from
the file; what the design fixes (the pairing of rotated dimensions, the null
key, softmax routing, activations) lives here and in the parts.

  architecture      "Buludra"
  vocab, width, max_positions (optional: the design has no limit, so 2^20 unless given)
  norm.eps          epsilon of every RMS norm (plain gains)
  logit_softcap     cap on the logits (null or absent: none)
  layers[i]         {type, mixer: {...}, mlp: {...} | null, weights_of: j | absent}
    attention       heads, kv_heads, dim, vdim, scale, q_temp: {coef, every} | absent   (q and k normed per head, no rotation)
    gla             heads, dim, vdim, tau; decay_rank (optional: the narrow size of the decay's two-step projection,
                    which otherwise the checkpoint's tensors give)
    parallel        left_scale, right_scale,
                    left:  heads, kv_heads, dim, vdim, scale, rot: {dims, base}   (rotated, unit norm, a null key)
                    right: heads, dim, vdim, gate_cap                             (matrix memory)
    mlp             {kind: "dense", ff}
                    {kind: "moe", expert: {ff}, router: {experts, top, groups: {count, keep} | absent}, shared: {ff} | absent}

Layer i's tensors start with "l<i>."; the block is pre-norm with two norms
(`norm1`, `norm2`); a norm (`final.norm`) and an untied head (`head`) end the
model.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .keys import ConfigError, opt_int, req_float, req_int, req_str
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Buludra"
MIXERS = ("attention", "gla", "parallel")


def _obj(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: missing config key: {key} (an object)")
    return v


def _positive(d: Mapping[str, Any], key: str, where: str) -> float:
    v = req_float(d, key)
    if not v > 0.0:
        raise ConfigError(f"{where}.{key} must be > 0, got {v}")
    return v


def _check_attention(m: Mapping[str, Any], where: str) -> None:
    for k in ("heads", "kv_heads", "dim", "vdim"):
        req_int(m, k)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: heads is not a multiple of kv_heads")
    _positive(m, "scale", where)


def _check_mlp(mlp: Any, w: str) -> None:
    if not isinstance(mlp, dict):
        raise ConfigError(f"{w}.mlp is neither null nor an object")
    kind = req_str(mlp, "kind")
    if kind == "dense":
        req_int(mlp, "ff")
        return
    if kind != "moe":
        raise ConfigError(f"{w}.mlp.kind is {kind!r}; known: dense, moe")
    req_int(_obj(mlp, "expert", w + ".mlp"), "ff")
    ro = _obj(mlp, "router", w + ".mlp")
    E, top = req_int(ro, "experts"), req_int(ro, "top")
    count = keep = 1
    if ro.get("groups") is not None:
        gr = _obj(ro, "groups", w + ".mlp.router")
        count, keep = req_int(gr, "count"), req_int(gr, "keep")
    if E % count or keep > count:
        raise ConfigError(f"{w}.mlp.router: {E} experts do not form {count} equal groups of which {keep} are kept")
    if top > keep * (E // count):
        raise ConfigError(f"{w}.mlp.router.top exceeds the experts of the kept groups")
    if mlp.get("shared") is not None:
        req_int(_obj(mlp, "shared", w + ".mlp"), "ff")


@dataclass(frozen=True)
class BuludraConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    logit_softcap: Optional[float]
    layers: tuple                       # of plain dictionaries as in config.json, checked
    has_max_positions: bool = False

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], generation: Mapping[str, Any] | None = None) -> "BuludraConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("missing config key: layers (a non-empty list)")
        mp = opt_int(d, "max_positions", None)
        cfg = cls(vocab=req_int(d, "vocab"), width=req_int(d, "width"), max_positions=mp if mp is not None else 1 << 20,
                  norm_eps=req_float(_obj(d, "norm", "config"), "eps"),
                  logit_softcap=_positive(d, "logit_softcap", "config") if d.get("logit_softcap") is not None else None,
                  layers=tuple(copy.deepcopy(layers)), has_max_positions=mp is not None)
        cfg.check()
        return cfg

    def check(self) -> None:
        if not self.norm_eps > 0.0:
            raise ConfigError(f"norm.eps must be > 0, got {self.norm_eps}")
        if self.max_positions < 1:
            raise ConfigError(f"max_positions must be >= 1, got {self.max_positions}")
        for i, L in enumerate(self.layers):
            w = f"layers[{i}]"
            if not isinstance(L, dict):
                raise ConfigError(f"{w} is not an object")
            kind = req_str(L, "type")
            if kind not in MIXERS:
                raise ConfigError(f"{w}.type is {kind!r}; known: {', '.join(MIXERS)}")
            m, wm = _obj(L, "mixer", w), w + ".mixer"
            if kind == "attention":
                _check_attention(m, wm)
                if m.get("q_temp") is not None:
                    qt = _obj(m, "q_temp", wm)
                    req_float(qt, "coef")
                    _positive(qt, "every", wm + ".q_temp")
            elif kind == "gla":
                for k in ("heads", "dim", "vdim"):
                    req_int(m, k)
                _positive(m, "tau", wm)
                opt_int(m, "decay_rank", None)
            else:
                a, r = _obj(m, "left", wm), _obj(m, "right", wm)
                req_float(m, "left_scale"), req_float(m, "right_scale")
                _check_attention(a, wm + ".left")
                rot = _obj(a, "rot", wm + ".left")
                dims = req_int(rot, "dims")
                if dims % 2 or dims > a["dim"]:
                    raise ConfigError(f"{wm}.left.rot.dims must be even and at most dim, got {dims}")
                _positive(rot, "base", wm + ".left.rot")
                for k in ("heads", "dim", "vdim"):
                    req_int(r, k)
                _positive(r, "gate_cap", wm + ".right")
            if L.get("mlp") is not None:
                _check_mlp(L["mlp"], w)
        for i, L in enumerate(self.layers):
            j = self.owner(i)
            if j != i and ({k: v for k, v in L.items() if k != "weights_of"}
                           != {k: v for k, v in self.layers[j].items() if k != "weights_of"}):
                raise ConfigError(f"layers[{i}] uses the weights of layers[{j}] but is not like it")

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = [i]
        while self.layers[i].get("weights_of") is not None:
            i = req_int(self.layers[i], "weights_of", 0)
            if i >= len(self.layers) or i in seen:
                raise ConfigError(f"layers[{seen[0]}].weights_of does not lead to a layer with tensors of its own")
            seen.append(i)
        return i

    def to_dict(self) -> dict[str, Any]:
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": copy.deepcopy(list(self.layers))}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.has_max_positions:
            d["max_positions"] = self.max_positions
        return d

    # ---------------------------------------------------------------- spec
    def _attention(self, m: Mapping[str, Any], p: str, extra: Mapping[str, Any]) -> PartSpec:
        return PartSpec("capped_attention", {
            "hidden_size": self.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
            "scale": float(m["scale"]), "eps": self.norm_eps, "pad_heads": True, "q": p + "q", "k": p + "k", "v": p + "v",
            "o": p + "o", **extra})

    def _mixer(self, i: int, L: Mapping[str, Any]) -> PartSpec:
        p = f"l{i}.mix."
        m = L["mixer"]
        memory = lambda kind, c, q, extra: PartSpec(kind, {
            "hidden_size": self.width, "heads": c["heads"], "dim": c["dim"], "vdim": c["vdim"], "eps": self.norm_eps,
            **{k: q + k for k in ("q", "k", "v", "g", "o", "norm")}, **extra})
        if L["type"] == "attention":
            qt = m.get("q_temp")
            return self._attention(m, p, {
                "qk_norm": True, "q_norm": p + "q.norm", "k_norm": p + "k.norm",
                "q_temp": {"coef": float(qt["coef"]), "every": float(qt["every"])} if qt else None})
        if L["type"] == "gla":
            return memory("gated_linear_attention", m, p, {"tau": float(m["tau"]), "rank": m.get("decay_rank"), "a1": p + "a1",
                                                           "a2": p + "a2", "a2_bias": p + "a2.b"})
        a, r = m["left"], m["right"]
        left = self._attention(a, p + "left.", {
            "qk_norm": "unit", "null_key": True,
            "rot": {"dims": int(a["rot"]["dims"]), "base": float(a["rot"]["base"]), "pairing": "half", "scaling": None}})
        q = p + "right."
        right = memory("matrix_memory", r, q, {"gate_cap": float(r["gate_cap"]), "i": q + "i", "i_bias": q + "i.b", "f": q + "f",
                                               "f_bias": q + "f.b"})
        return PartSpec("parallel_mixers", {"hidden_size": self.width, "branches": (left, right),
                                            "scales": (float(m["left_scale"]), float(m["right_scale"]))})

    def _ffn(self, i: int, mlp: Mapping[str, Any]) -> PartSpec:
        p = f"l{i}.mlp."
        if mlp["kind"] == "dense":
            return PartSpec("swiglu_dense", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "gate": p + "gate",
                                             "up": p + "up", "down": p + "down"})
        ro = mlp["router"]
        gr = ro.get("groups") or {"count": 1, "keep": 1}
        shared = mlp.get("shared")
        return PartSpec("group_router_experts", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "experts": ro["experts"], "top": ro["top"],
            "groups": gr["count"], "keep": gr["keep"], "scores": "softmax", "group_score": "max", "limit": None,
            "router": p + "router", "expert_prefix": p + "e", "shared": shared["ff"] if shared else None,
            "shared_prefix": p + "shared.", "shared_gate": p + "shared.sg"})

    def model_spec(self) -> ModelSpec:
        owners = sorted({self.owner(i) for i in range(len(self.layers))})
        layers = []
        for i in owners:
            L, p = self.layers[i], f"l{i}."
            norm = lambda name: PartSpec("rmsnorm", {"eps": self.norm_eps, "dim": self.width, "name": name})
            mlp = L.get("mlp")
            norms = {"mixer": norm(p + "norm1")}
            if mlp is not None:
                norms["ffn"] = norm(p + "norm2")
            layers.append(LayerSpec(block=PartSpec("prenorm_residual", {}), mixer=self._mixer(i, L),
                                    ffn=self._ffn(i, mlp) if mlp is not None else None, norms=norms, prefix=p))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, max_positions=self.max_positions,
            layers=tuple(layers),
            schedule=tuple(ScheduleEntry(owners.index(self.owner(i))) for i in range(len(self.layers))),
            embedding=PartSpec("token_embedding", {"name": "embed", "vocab_size": self.vocab, "dim": self.width}),
            final_norm=PartSpec("rmsnorm", {"eps": self.norm_eps, "dim": self.width, "name": "final.norm"}),
            head=PartSpec("linear_head", {"tied": False, "name": "head", "vocab_size": self.vocab, "dim": self.width,
                                          "logit_softcap": self.logit_softcap}))
        spec.validate()
        return spec
