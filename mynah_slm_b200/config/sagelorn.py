"""Typed configuration of the Sagelorn design, read from its config.json.

A small decoder-only model whose layers are listed one by one: `layers[i]`
names the layer's mixer (`type`), the mixer's sizes (`mixer`) and its
feed-forward (`mlp`, or null for none). The residual stream is read as it is:
every norm stands behind its sublayer. Every size and every constant that can
differ between two models of the design is read from the file; what the design
fixes (which mixer pairs rotated dimensions how, sinks, the gates' and experts'
activations, weights on the experts' inputs) lives here and in the parts.

  architecture      "Sagelorn"
  vocab, width, max_positions (optional: the design has no limit, so 2^20 unless given)
  embedding.bigram  {buckets, mul_prev, mul_cur}: a second embedding table [buckets + 1, width] looked up by a
                    token and the one before it
  norm.eps          epsilon of every RMS norm (the layers' gains are stored around zero: 1 + w)
  logit_scale       the logits are multiplied by it
  layers[i]         {type, mixer: {...}, mlp: {...} | null}
    attention         heads, kv_heads, dim, vdim, scale, rot: {dims, base, scaling?}, mask: {size} | absent, kv_from?: j
                      (q and k normed over the whole projection, a sink a head, pairs (i, i + dims/2); kv_from: the layer
                      has no key and value projections and reads layer j's keys and values through a mask of its own)
    latent_attention  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot: {dims, base, scaling?}, mask: {size} | absent
                      (a gate for every value, pairs (2i, 2i+1); q_rank absent: the checkpoint's tensors give it)
    retention         heads, dim, vdim, decay: [per head]   (no rotation)
    rot.scaling       {factor, low, high, original}: frequencies scaled by wavelength
    mlp               {kind: "dense", ff}
                      {kind: "moe", expert: {ff}, router: {experts, top}, shared: {ff} | absent}

Layer i's tensors start with "l<i>."; the block norms each sublayer's output
(`norm1`, `norm2`); a norm (`final.norm`) and an untied head (`head`) end the
model.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .keys import ConfigError, opt_int, req_float, req_int, req_str
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Sagelorn"
MIXERS = ("attention", "latent_attention", "retention")


def _obj(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: missing config key: {key} (an object)")
    return v


def _check_rot(m: Mapping[str, Any], limit: int, where: str) -> None:
    rot = _obj(m, "rot", where)
    dims = req_int(rot, "dims")
    if dims % 2 or dims > limit:
        raise ConfigError(f"{where}.rot.dims must be even and at most {limit}, got {dims}")
    if not req_float(rot, "base") > 0.0:
        raise ConfigError(f"{where}.rot.base must be > 0")
    if rot.get("scaling") is not None:
        sc = _obj(rot, "scaling", where + ".rot")
        for k in ("factor", "low", "high", "original"):
            if not req_float(sc, k) > 0.0:
                raise ConfigError(f"{where}.rot.scaling.{k} must be > 0")
        if float(sc["low"]) == float(sc["high"]):
            raise ConfigError(f"{where}.rot.scaling: low and high are equal")


def _rot_spec(rot: Mapping[str, Any], pairing: str) -> dict:
    sc = rot.get("scaling")
    return {"dims": int(rot["dims"]), "base": float(rot["base"]), "pairing": pairing,
            "scaling": {"kind": "wavelength", **{k: float(sc[k]) for k in ("factor", "low", "high", "original")}} if sc else None}


def _window(m: Mapping[str, Any]) -> Optional[int]:
    return m["mask"]["size"] if m.get("mask") is not None else None


@dataclass(frozen=True)
class SagelornConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    logit_scale: float
    bigram: Mapping[str, int]           # buckets, mul_prev, mul_cur
    layers: tuple                       # of plain dictionaries as in config.json, checked
    has_max_positions: bool = False

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], generation: Mapping[str, Any] | None = None) -> "SagelornConfig":
        layers = d.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("missing config key: layers (a non-empty list)")
        mp = opt_int(d, "max_positions", None)
        bg = _obj(_obj(d, "embedding", "config"), "bigram", "embedding")
        cfg = cls(vocab=req_int(d, "vocab"), width=req_int(d, "width"), max_positions=mp if mp is not None else 1 << 20,
                  norm_eps=req_float(_obj(d, "norm", "config"), "eps"), logit_scale=req_float(d, "logit_scale"),
                  bigram={"buckets": req_int(bg, "buckets"), "mul_prev": req_int(bg, "mul_prev", 0), "mul_cur": req_int(bg, "mul_cur", 0)},
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
            m = _obj(L, "mixer", w)
            getattr(self, "_check_" + kind)(i, m, w + ".mixer")
            if L.get("mlp") is not None:
                self._check_mlp(L["mlp"], w + ".mlp")

    @staticmethod
    def _check_mask(m: Mapping[str, Any], where: str) -> None:
        if m.get("mask") is not None:
            req_int(_obj(m, "mask", where), "size")

    def _check_attention(self, i: int, m: Mapping[str, Any], where: str) -> None:
        for k in ("heads", "kv_heads", "dim", "vdim"):
            req_int(m, k)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: heads is not a multiple of kv_heads")
        if not req_float(m, "scale") > 0.0:
            raise ConfigError(f"{where}.scale must be > 0")
        _check_rot(m, m["dim"], where)
        self._check_mask(m, where)
        j = opt_int(m, "kv_from", None)
        if j is None:
            return
        if not 0 <= j < i:
            raise ConfigError(f"{where}.kv_from names layer {j}, which does not run before layer {i}")
        S = self.layers[j]
        if S.get("type") != "attention" or S["mixer"].get("kv_from") is not None:
            raise ConfigError(f"{where}.kv_from names layer {j}, which keeps no keys and values of its own")
        for k in ("kv_heads", "dim", "vdim", "rot"):
            if S["mixer"].get(k) != m.get(k):
                raise ConfigError(f"{where}.{k} differs from that of layer {j}, whose keys and values it reads")

    def _check_latent_attention(self, i: int, m: Mapping[str, Any], where: str) -> None:
        for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"):
            req_int(m, k)
        if m.get("q_rank") is not None:
            req_int(m, "q_rank")
        if not req_float(m, "scale") > 0.0:
            raise ConfigError(f"{where}.scale must be > 0")
        _check_rot(m, m["rot_dim"], where)
        self._check_mask(m, where)

    def _check_retention(self, i: int, m: Mapping[str, Any], where: str) -> None:
        for k in ("heads", "dim", "vdim"):
            req_int(m, k)
        decay = m.get("decay")
        if (not isinstance(decay, list) or len(decay) != m["heads"]
                or not all(isinstance(x, (int, float)) and not isinstance(x, bool) and x >= 0 for x in decay)):
            raise ConfigError(f"{where}.decay must list one number per head, none of them negative")

    @staticmethod
    def _check_mlp(mlp: Any, where: str) -> None:
        if not isinstance(mlp, dict):
            raise ConfigError(f"{where} is neither null nor an object")
        kind = req_str(mlp, "kind")
        if kind == "dense":
            req_int(mlp, "ff")
        elif kind == "moe":
            req_int(_obj(mlp, "expert", where), "ff")
            ro = _obj(mlp, "router", where)
            if req_int(ro, "top") > req_int(ro, "experts"):
                raise ConfigError(f"{where}.router.top exceeds the number of experts")
            if mlp.get("shared") is not None:
                req_int(_obj(mlp, "shared", where), "ff")
        else:
            raise ConfigError(f"{where}.kind is {kind!r}; known: dense, moe")

    def to_dict(self) -> dict[str, Any]:
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "embedding": {"bigram": dict(self.bigram)},
             "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers))}
        if self.has_max_positions:
            d["max_positions"] = self.max_positions
        return d

    # ---------------------------------------------------------------- spec
    def _mixer(self, i: int, L: Mapping[str, Any]) -> PartSpec:
        p, m = f"l{i}.mix.", L["mixer"]
        names = lambda *keys: {k: p + k for k in keys}
        common = {"hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "eps": self.norm_eps,
                  "output": "fp32"}
        if L["type"] == "attention":
            return PartSpec("projnorm_attention", {
                **common, "kv_heads": m["kv_heads"], "scale": float(m["scale"]), "rot": _rot_spec(m["rot"], "half"),
                "window": _window(m), "value_norm": False, "own_kv": m.get("kv_from") is None, "pad_heads": True, "sink": p + "sink",
                "q_norm": p + "q.norm", "k_norm": p + "k.norm", **names("q", "k", "v", "o")})
        if L["type"] == "latent_attention":
            return PartSpec("latent_attention", {
                **common, "rot_dim": m["rot_dim"], "kv_rank": m["kv_rank"], "q_rank": m["q_rank"] if m.get("q_rank") is not None else -1,
                "scale": float(m["scale"]), "rot": _rot_spec(m["rot"], "interleaved"), "window": _window(m), "own_kv": True,
                "pad_heads": True, "gate": p + "g", "gate_kind": "value", "q": p + "uq", "dq_norm": p + "dq.norm",
                "dkv_norm": p + "dkv.norm", **names("dq", "dkv", "uk", "uv", "o")})
        return PartSpec("retention", {**common, "decay": [float(x) for x in m["decay"]], "rot": None, **names("q", "k", "v", "g", "o")})

    def _ffn(self, i: int, mlp: Mapping[str, Any]) -> PartSpec:
        p = f"l{i}.mlp."
        if mlp["kind"] == "dense":
            return PartSpec("swiglu_dense", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "output": "fp32", "gate": p + "gate",
                                             "up": p + "up", "down": p + "down"})
        ro, shared = mlp["router"], mlp.get("shared")
        return PartSpec("group_router_experts", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "experts": ro["experts"], "top": ro["top"],
            "activation": "relu2", "weights_on": "input", "output": "fp32", "router": p + "router", "expert_prefix": p + "e",
            "shared": shared["ff"] if shared else None, "shared_prefix": p + "shared."})

    def model_spec(self) -> ModelSpec:
        layers, schedule = [], []
        for i, L in enumerate(self.layers):
            p, mlp = f"l{i}.", L.get("mlp")
            norm = lambda name: PartSpec("rmsnorm_offset", {"eps": self.norm_eps, "dim": self.width, "name": name})
            norms = {"mixer": norm(p + "norm1")}
            if mlp is not None:
                norms["ffn"] = norm(p + "norm2")
            layers.append(LayerSpec(block=PartSpec("postnorm_residual", {"hidden_size": self.width}), mixer=self._mixer(i, L),
                                    ffn=self._ffn(i, mlp) if mlp is not None else None, norms=norms, prefix=p))
            # one run a layer, in order: schedule index == layer index
            schedule.append(ScheduleEntry(i, cache_from=L["mixer"].get("kv_from")))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, max_positions=self.max_positions,
            layers=tuple(layers), schedule=tuple(schedule),
            embedding=PartSpec("token_pair_embedding", {"name": "embed", "pair_name": "bigram", "vocab_size": self.vocab,
                                                        "dim": self.width, **self.bigram}),
            final_norm=PartSpec("rmsnorm_offset", {"eps": self.norm_eps, "dim": self.width, "name": "final.norm"}),
            head=PartSpec("linear_head", {"tied": False, "name": "head", "vocab_size": self.vocab, "dim": self.width,
                                          "logit_scale": self.logit_scale}))
        spec.validate()
        return spec
