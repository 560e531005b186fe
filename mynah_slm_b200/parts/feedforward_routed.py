"""Feed-forwards of several small experts, of which every token uses `top`.

`table_routed_experts` picks without a router: a table [vocab, top] gives each token id its experts (the
entries of a row differ), and each counts 1/top.

An expert, with h its input (no biases):

  g = min(W_gate h, limit),   u = clamp(W_up h, -limit, limit)
  y = g * sigmoid(alpha g) * (u + 1),   out = W_down y

The step's (token, choice) pairs are sorted by expert on the device and the two
products run tile by tile over rows that share an expert (`csrc/moe.cu`); the
experts' matrices are stacked at bind time.

Parameters: hidden_size, intermediate_size (of one expert), experts, top, limit,
alpha (1.702 unless given), vocab_size, table (tensor name) and expert_prefix:
expert e's tensors are `<expert_prefix><e>.gate`, `.up` and `.down`.

`router_experts` picks with a learned router:

  z = W_r h + b_r  (fp32);  the `top` largest z (the lower index wins a tie);
  their weights are softmax over the chosen z alone
  expert:  out = W_down act(W_up h),  act the exact (erf) GELU, no gate, no biases
  result = sum over the chosen of weight * expert(h),  fp32 rows (not rounded to the activation type)

Parameters: hidden_size, intermediate_size, experts, top, activation
("gelu_erf"), router, router_bias (tensor names) and expert_prefix: expert e's
tensors are `<expert_prefix><e>.up` and `.down`.

`group_router_experts` picks with sigmoid scores, a correction and groups:

  s = sigmoid(W_r h)  (fp32);  the choice goes by s + correction
  the experts form `groups` equal groups of neighbours; a group counts the sum of its two largest choice scores;
  only experts of the `keep` best groups can be chosen (the lower index wins every tie)
  the `top` largest choice scores among them; each counts s (without the correction) * weight_scale, not renormalised
  expert: the clamped-gate expert of `table_routed_experts` (limit, alpha)

Variants, chosen by parameters: scores "softmax" (over all experts, instead of the sigmoid); group_score "max" (a group
counts its largest choice score); correction None; limit None: the expert is W_down (silu(W_gate h) * (W_up h)). With
`shared`, a feed-forward of that last form that every token passes (its intermediate size, and its tensors'
`shared_prefix`), multiplied by sigmoid(w . h), one number a token (w: `shared_gate`; None: not multiplied), is added.
activation "relu2": expert and shared expert are W_down relu(W_up h)^2 (`.up` and `.down`; no gate matrix). weights_on
"input": a token's weight multiplies its expert's input instead of its output (one-matrix experts; the shared expert reads h as it
is). Such a shared expert of the experts' own size runs as one more expert of small steps; else its two products are ordinary
ones.

Parameters: hidden_size, intermediate_size, experts, top, groups (1), keep (= groups), weight_scale (1), limit, alpha
(1.702), scores ("sigmoid"), group_score ("top2"), activation ("gated"), weights_on ("output"), output ("act", or "fp32": the sum
is not rounded), router, correction (tensor names), expert_prefix, and optionally shared, shared_prefix, shared_gate.
"""
from __future__ import annotations

from typing import Mapping

import torch

from ..config.keys import ConfigError
from ..ops import kernels
from .base import FeedForward, TensorSpec, register_ffn


class TableRoutedExperts(FeedForward):
    def __init__(self, spec):
        super().__init__(spec)
        g = lambda k: int(spec[k])
        self.D, self.F, self.E, self.top, self.V = (g("hidden_size"), g("intermediate_size"), g("experts"), g("top"),
                                                    g("vocab_size"))
        self.limit = float(spec["limit"])
        self.alpha = float(spec.get("alpha", 1.702))
        self.table_name = str(spec["table"])
        self.prefix = str(spec["expert_prefix"])
        if not 1 <= self.top <= self.E:
            raise ConfigError(f"table_routed_experts: top {self.top} does not fit {self.E} experts")
        if self.E > 1024:
            raise ConfigError(f"table_routed_experts: {self.E} experts exceed the 1024 that the routing kernel counts")

    def _name(self, e: int, which: str) -> str:
        return f"{self.prefix}{e}.{which}"

    def tensor_specs(self) -> list[TensorSpec]:
        specs = [TensorSpec(self.table_name, (self.V, self.top), role="table", init=f"distinct:{self.E}")]
        for e in range(self.E):
            specs += [TensorSpec(self._name(e, "gate"), (self.F, self.D)), TensorSpec(self._name(e, "up"), (self.F, self.D)),
                      TensorSpec(self._name(e, "down"), (self.D, self.F))]
        return specs

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        self.table = tensors[self.table_name].contiguous()
        self.w_gu = torch.stack([torch.stack([tensors[self._name(e, "gate")], tensors[self._name(e, "up")]])
                                 for e in range(self.E)]).contiguous()
        self.w_down = torch.stack([tensors[self._name(e, "down")] for e in range(self.E)]).contiguous()

    def streamed_tensors(self) -> list:
        return []          # a step reads only the experts its tokens pick

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return kernels.moe_table_ffn(h, self.table, self.w_gu, self.w_down, ctx, self.top, self.limit, self.alpha)


register_ffn("table_routed_experts", TableRoutedExperts)


class RouterExperts(FeedForward):
    def __init__(self, spec):
        super().__init__(spec)
        g = lambda k: int(spec[k])
        self.D, self.F, self.E, self.top = g("hidden_size"), g("intermediate_size"), g("experts"), g("top")
        self.router_name, self.bias_name = str(spec["router"]), str(spec["router_bias"])
        self.prefix = str(spec["expert_prefix"])
        if spec.get("activation", "gelu_erf") != "gelu_erf":
            raise ConfigError(f"router_experts: activation {spec.get('activation')!r} is not built in (gelu_erf)")
        if not 1 <= self.top <= self.E:
            raise ConfigError(f"router_experts: top {self.top} does not fit {self.E} experts")
        if self.E > 1024:
            raise ConfigError(f"router_experts: {self.E} experts exceed the 1024 that the routing kernel counts")

    def _name(self, e: int, which: str) -> str:
        return f"{self.prefix}{e}.{which}"

    def tensor_specs(self) -> list[TensorSpec]:
        specs = [TensorSpec(self.router_name, (self.E, self.D), std=0.3),
                 TensorSpec(self.bias_name, (self.E,), role="gain", init="normal", std=0.3)]
        for e in range(self.E):
            specs += [TensorSpec(self._name(e, "up"), (self.F, self.D)), TensorSpec(self._name(e, "down"), (self.D, self.F))]
        return specs

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        self.w_router = tensors[self.router_name].contiguous()
        self.b_router = tensors[self.bias_name].contiguous()
        self.w_up = torch.stack([tensors[self._name(e, "up")] for e in range(self.E)]).contiguous()
        self.w_down = torch.stack([tensors[self._name(e, "down")] for e in range(self.E)]).contiguous()

    def streamed_tensors(self) -> list:
        return [self.w_router]          # of the experts a step reads only those its tokens pick

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return kernels.moe_router_ffn(h, self.w_router, self.b_router, self.w_up, self.w_down, ctx, self.top)


register_ffn("router_experts", RouterExperts)


class GroupRouterExperts(FeedForward):
    def __init__(self, spec):
        super().__init__(spec)
        g = lambda k: int(spec[k])
        self.D, self.F, self.E, self.top = g("hidden_size"), g("intermediate_size"), g("experts"), g("top")
        self.groups = int(spec.get("groups", 1))
        self.keep = int(spec.get("keep", self.groups))
        self.weight_scale = float(spec.get("weight_scale", 1.0))
        self.limit = None if spec.get("limit") is None else float(spec["limit"])
        self.alpha = float(spec.get("alpha", 1.702))
        self.scores, self.group_score = str(spec.get("scores", "sigmoid")), str(spec.get("group_score", "top2"))
        self.router_name = str(spec["router"])
        self.correction_name = str(spec["correction"]) if spec.get("correction") is not None else None
        self.FS = int(spec.get("shared") or 0)
        self.shared_prefix = str(spec["shared_prefix"]) if self.FS else ""
        self.shared_gate = str(spec["shared_gate"]) if self.FS and spec.get("shared_gate") is not None else None
        self.relu2 = str(spec.get("activation", "gated")) == "relu2"
        self.weights_on = str(spec.get("weights_on", "output"))
        self.out_dtype = torch.float32 if str(spec.get("output", "act")) == "fp32" else None
        if spec.get("activation", "gated") not in ("gated", "relu2") or self.weights_on not in ("output", "input"):
            raise ConfigError("group_router_experts: unknown activation or place of the weights")
        if self.weights_on == "input" and not self.relu2:
            raise ConfigError("group_router_experts: weights on the input go with experts of one matrix before the activation")
        if self.relu2 and self.limit is not None:
            raise ConfigError("group_router_experts: the squared relu has no limit")
        if self.scores not in ("sigmoid", "softmax") or self.group_score not in ("top2", "max"):
            raise ConfigError(f"group_router_experts: scores {self.scores!r} or group score {self.group_score!r} is not built in")
        self.prefix = str(spec["expert_prefix"])
        if self.E + (1 if self.FS else 0) > 1024:
            raise ConfigError(f"group_router_experts: {self.E} experts exceed the 1024 that the routing kernel counts")
        if self.groups < 1 or self.E % self.groups or not 1 <= self.keep <= self.groups:
            raise ConfigError(f"group_router_experts: {self.E} experts do not form {self.groups} equal groups of which "
                              f"{self.keep} are kept")
        if not 1 <= self.top <= self.keep * (self.E // self.groups):
            raise ConfigError(f"group_router_experts: top {self.top} does not fit the experts of {self.keep} kept groups")

    def _name(self, e: int, which: str) -> str:
        return f"{self.prefix}{e}.{which}"

    def tensor_specs(self) -> list[TensorSpec]:
        specs = [TensorSpec(self.router_name, (self.E, self.D), std=0.3)]
        if self.correction_name is not None:
            specs.append(TensorSpec(self.correction_name, (self.E,), role="gain", init="normal", std=0.1))
        if self.FS:
            p = self.shared_prefix
            specs += [TensorSpec(p + which, (self.FS, self.D)) for which in self._inner()]
            specs.append(TensorSpec(p + "down", (self.D, self.FS)))
            if self.shared_gate is not None:
                specs.append(TensorSpec(self.shared_gate, (1, self.D)))
        for e in range(self.E):
            specs += [TensorSpec(self._name(e, which), (self.F, self.D)) for which in self._inner()]
            specs.append(TensorSpec(self._name(e, "down"), (self.D, self.F)))
        return specs

    def _inner(self) -> tuple[str, ...]:
        """The matrices before the activation."""
        return ("up",) if self.relu2 else ("gate", "up")

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        self.w_router = tensors[self.router_name].contiguous()
        self.correction = tensors[self.correction_name].contiguous() if self.correction_name is not None else None
        self.w_shared = None
        if self.FS:
            p = self.shared_prefix
            if self.shared_gate is not None:
                self.w_router = torch.cat([self.w_router, tensors[self.shared_gate]], dim=0).contiguous()
            self.w_shared = torch.cat([tensors[p + which] for which in self._inner()], dim=0).contiguous()
            self.w_shared_down = tensors[p + "down"]
        names = [f"{self.prefix}{e}." for e in range(self.E)]
        # a shared expert of the experts' own form and size, without a gate, lies behind them
        self.shared_in_stack = bool(self.FS) and self.FS == self.F and self.weights_on == "input" and self.shared_gate is None
        if self.shared_in_stack:
            names.append(self.shared_prefix)
        if self.relu2:
            self.w_gu = torch.stack([tensors[n + "up"] for n in names]).contiguous()
        else:
            self.w_gu = torch.stack([torch.stack([tensors[n + "gate"], tensors[n + "up"]]) for n in names]).contiguous()
        self.w_down = torch.stack([tensors[n + "down"] for n in names]).contiguous()
        if self.shared_in_stack:                                 # one copy of it
            self.w_shared, self.w_shared_down = self.w_gu[self.E], self.w_down[self.E]

    def streamed_tensors(self) -> list:
        # of the experts a step reads only those its tokens pick
        return [self.w_router] + ([self.w_shared, self.w_shared_down] if self.FS else [])

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        shared, w_gu, w_down = None, self.w_gu, self.w_down
        in_stack = self.shared_in_stack and not kernels.moe_runs_grouped(h.shape[0], self.top + 1, self.E + 1, self.D, self.F, h.dtype)
        if self.FS and not in_stack:
            inner = kernels.linear_relu2 if self.relu2 else kernels.linear_swiglu
            shared = kernels.linear(inner(h, self.w_shared), self.w_shared_down, out_dtype=torch.float32)
            w_gu, w_down = w_gu[: self.E], w_down[: self.E]
        return kernels.moe_group_router_ffn(h, self.w_router, self.correction, w_gu, w_down, ctx, self.top,
                                            self.groups, self.keep, self.weight_scale, self.limit, self.alpha, self.scores,
                                            self.group_score, shared, "relu2" if self.relu2 else "gated", self.weights_on,
                                            self.shared_gate is not None, in_stack, self.out_dtype)


register_ffn("group_router_experts", GroupRouterExperts)
