"""Linear attention with learned decays, as a mixer in two kinds. With h the mixer's input, per head:

`gated_linear_attention` (GLA: Yang, Wang, Shen, Panda, Kim, "Gated Linear Attention Transformers with
Hardware-Efficient Training", 2023)

  q = W_q h * dim^(-1/2), k = W_k h (heads x dim), v = W_v h (heads x vdim)
  z = W_a2 (W_a1 h) + b   (heads x dim);   a = sigmoid(z)^(1/tau), a decay a key channel
  S <- diag(a) S + k v^T;   o = S^T q
  out = W_o [o / rms(o) * w * silu(W_g h)]          w of vdim values, shared by the heads

`matrix_memory` (the mLSTM of xLSTM: Beck, Poeppel et al., "xLSTM: Extended Long Short-Term Memory", 2024)

  q, k, v as above;   i = cap tanh((W_i h + b_i) / cap),   f = log sigmoid(cap tanh((W_f h + b_f) / cap))
  m' = max(f + m, i) from m = 0;   S <- e^(f + m - m') S + e^(i - m') k v^T;   n likewise with k alone
  o = S^T q / (max(|n . q|, e^(-m')) + 1e-6)
  out = W_o [o / rms(o) * w * sigmoid(W_g h)]       w of heads x vdim values

State (fp32, from zero): S [heads, dim, vdim]; the matrix memory also n [heads, dim] and m [heads]. All projections of
h run as one product; the recurrence, the norm and the gate are one kernel launch in a decode step and three in a
bfloat16 prompt step (`csrc/gated_memory.cu`). rms is over the head's vdim values, with eps inside the root.

Parameters: hidden_size, heads, dim, vdim, eps, and the tensors' names q, k, v, g, o, norm; for the first also tau, a1, a2,
a2_bias and rank (None: what the checkpoint's tensors have), for the second gate_cap, i, i_bias, f, f_bias.

Both offer the two halves of their work to a mixer that shares its products (`in_weight`, `heads`, `out_weight`).
"""
from __future__ import annotations

from typing import Mapping

import torch

from ..config.keys import ConfigError
from ..ops import kernels
from .base import CacheView, Mixer, StateRequest, TensorSpec, register_mixer


class _GatedMemory(Mixer):
    kind = ""
    shares_products = True

    def __init__(self, spec):
        super().__init__(spec)
        g = lambda k: int(spec[k])
        self.D, self.H, self.dim, self.vd = g("hidden_size"), g("heads"), g("dim"), g("vdim")
        self.eps = float(spec["eps"])
        self.out_scale = 1.0                  # a factor on the output, formed with the norm's weight when the weights are bound
        self.tau = self.cap = 1.0
        if self.dim > 512 or self.vd > 512:
            raise ConfigError(f"{spec.kind}: heads of {self.dim} x {self.vd} exceed the 512 that the recurrence kernel stages")

    def _pieces(self, tensors) -> list[tuple[str, torch.Tensor]]:
        raise NotImplementedError

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        n = self.names
        self.at: dict[str, int] = {}
        parts, row = [], 0
        for name, w in self._pieces(tensors):        # every piece starts at a multiple of 8 rows of the stacked matrix
            self.at[name] = row
            parts.append(w)
            row += w.shape[0]
            if row % 8:
                parts.append(torch.zeros((8 - row % 8, self.D), dtype=w.dtype, device=w.device))
                row += 8 - row % 8
        self.in_weight = torch.cat(parts, dim=0).contiguous()
        self.out_weight = tensors[n["o"]]
        self.out_cols = self.H * self.vd
        w = tensors[n["norm"]].to(torch.float32)
        if w.numel() == self.vd and self.H > 1:
            w = w.repeat(self.H)
        self.w_norm = (w * self.out_scale).contiguous()
        self.w2 = None
        self.runtime = runtime

    def streamed_tensors(self) -> list:
        return [t for t in (self.in_weight, self.out_weight) if t is not None]

    def heads(self, p: torch.Tensor, out: torch.Tensor, ctx, cache: CacheView) -> None:
        """The mixer between its two products: p [T, in_weight rows] -> out[:, :out_cols]."""
        kernels.gated_memory(self.kind, p, self.at, self.w2, self.bias, self.w_norm, float(self.dim) ** -0.5, cache.state, out,
                             ctx, self.H, self.dim, self.vd, self.eps, self.tau, self.cap)

    def forward(self, h: torch.Tensor, ctx, cache: CacheView) -> torch.Tensor:
        p = kernels.linear(h, self.in_weight)
        out = torch.empty((p.shape[0], self.out_cols), dtype=p.dtype, device=p.device)
        self.heads(p, out, ctx, cache)
        return kernels.linear(out, self.out_weight)


class GatedLinearAttention(_GatedMemory):
    kind = "gla"

    def __init__(self, spec):
        super().__init__(spec)
        self.tau = float(spec["tau"])
        self.rank = -1 if spec.get("rank") is None else int(spec["rank"])
        self.names = {k: str(spec[k]) for k in ("q", "k", "v", "g", "o", "norm", "a1", "a2", "a2_bias")}
        if not self.tau > 0.0:
            raise ConfigError("gated_linear_attention: tau must be positive")

    def tensor_specs(self) -> list[TensorSpec]:
        n, H, D, dim, vd = self.names, self.H, self.D, self.dim, self.vd
        return [TensorSpec(n["q"], (H * dim, D)), TensorSpec(n["k"], (H * dim, D)), TensorSpec(n["v"], (H * vd, D)),
                TensorSpec(n["g"], (H * vd, D)), TensorSpec(n["o"], (D, H * vd)),
                TensorSpec(n["norm"], (vd,), role="gain", init="gain", std=0.1),
                TensorSpec(n["a1"], (self.rank, D), free_size=16), TensorSpec(n["a2"], (H * dim, self.rank), std=0.2, free_size=16),
                TensorSpec(n["a2_bias"], (H * dim,), role="gain", init="normal", std=0.5)]

    def _pieces(self, tensors):
        n = self.names
        return [(k, tensors[n[k]]) for k in ("q", "k", "v", "g")] + [("a", tensors[n["a1"]])]

    def bind(self, tensors, runtime) -> None:
        n = self.names
        if tensors[n["a2"]].shape[1] != tensors[n["a1"]].shape[0]:
            raise ConfigError(f"gated_linear_attention: {n['a1']} and {n['a2']} do not agree on the narrow size")
        super().bind(tensors, runtime)
        self.w2 = tensors[n["a2"]].contiguous()
        self.bias = tensors[n["a2_bias"]].to(torch.float32).contiguous()

    def state_request(self):
        return {"S": StateRequest((self.H, self.dim, self.vd), torch.float32)}


class MatrixMemory(_GatedMemory):
    kind = "mlstm"

    def __init__(self, spec):
        super().__init__(spec)
        self.cap = float(spec["gate_cap"])
        self.names = {k: str(spec[k]) for k in ("q", "k", "v", "g", "o", "norm", "i", "i_bias", "f", "f_bias")}
        if not self.cap > 0.0:
            raise ConfigError("matrix_memory: gate_cap must be positive")

    def tensor_specs(self) -> list[TensorSpec]:
        n, H, D, dim, vd = self.names, self.H, self.D, self.dim, self.vd
        return [TensorSpec(n["q"], (H * dim, D)), TensorSpec(n["k"], (H * dim, D)), TensorSpec(n["v"], (H * vd, D)),
                TensorSpec(n["g"], (H * vd, D)), TensorSpec(n["o"], (D, H * vd)),
                TensorSpec(n["norm"], (H * vd,), role="gain", init="gain", std=0.1),
                TensorSpec(n["i"], (H, D)), TensorSpec(n["i_bias"], (H,), role="gain", init="normal", std=1.0),
                TensorSpec(n["f"], (H, D)), TensorSpec(n["f_bias"], (H,), role="gain", init="normal", std=1.0)]

    def _pieces(self, tensors):
        return [(k, tensors[self.names[k]]) for k in ("q", "k", "v", "g", "i", "f")]

    def bind(self, tensors, runtime) -> None:
        super().bind(tensors, runtime)
        self.bias = torch.cat([tensors[self.names[k]].to(torch.float32) for k in ("i_bias", "f_bias")]).contiguous()

    def state_request(self):
        return {"S": StateRequest((self.H, self.dim, self.vd), torch.float32), "n": StateRequest((self.H, self.dim), torch.float32),
                "m": StateRequest((self.H,), torch.float32)}


register_mixer("gated_linear_attention", GatedLinearAttention)
register_mixer("matrix_memory", MatrixMemory)
