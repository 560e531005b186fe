"""Dense gated feed-forward (SwiGLU).

x -> W_down . (silu(W_gate . x) * (W_up . x)), no bias (mynah-slm
src/arch_qwen3.c:229-234, src/kernels.c:193-205). Parameters: hidden_size,
intermediate_size, activation (only "silu" is built), and either prefix (the
tensors are then <prefix>gate_proj.weight and so on) or the tensors' names gate,
up and down; `output`: "act" (the default: rows in the run's activation type) or
"fp32" (unrounded, for a norm that follows the sublayer). Gate and up are
kept as one fused matrix [2 * intermediate, hidden], gate rows first, so a
step is two products instead of three.
"""
from __future__ import annotations

from typing import Mapping

import torch

from ..config.keys import ConfigError
from ..ops import kernels
from .base import FeedForward, TensorSpec, register_ffn


class SwiGLUDense(FeedForward):
    accepts_normed = True        # its first product can compute the norm on its way

    def __init__(self, spec):
        super().__init__(spec)
        self.D = int(spec["hidden_size"])
        self.F = int(spec["intermediate_size"])
        if spec.get("prefix") is not None:
            self.names = {k: f"{spec['prefix']}{k}_proj.weight" for k in ("gate", "up", "down")}
        else:
            self.names = {k: str(spec[k]) for k in ("gate", "up", "down")}
        act = spec.get("activation", "silu")
        if act != "silu":
            raise ConfigError(f"swiglu_dense: activation {act!r} is not supported (only 'silu')")
        self.out_dtype = torch.float32 if str(spec.get("output", "act")) == "fp32" else None
        self.w_gate_up = self.w_down = None

    def tensor_specs(self) -> list[TensorSpec]:
        n = self.names
        return [TensorSpec(n["gate"], (self.F, self.D)), TensorSpec(n["up"], (self.F, self.D)), TensorSpec(n["down"], (self.D, self.F))]

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        n = self.names
        self.w_gate_up = torch.cat([tensors[n["gate"]], tensors[n["up"]]], dim=0).contiguous()
        self.w_down = tensors[n["down"]]

    def streamed_tensors(self) -> list:
        return [self.w_gate_up, self.w_down]

    def forward(self, h: torch.Tensor, ctx) -> torch.Tensor:
        return kernels.linear(kernels.linear_swiglu(h, self.w_gate_up), self.w_down, out_dtype=self.out_dtype)


register_ffn("swiglu_dense", SwiGLUDense)
