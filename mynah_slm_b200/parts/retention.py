"""Retention: linear attention with a fixed decay per head, no softmax and no
denominator.

With h the mixer's input (`csrc/retention.cu` states the recurrence):

  q = W_q h, k = W_k h   (heads x dim),   v = W_v h   (heads x vdim);   no biases
  q and k are rotated (the position part's pairing and tables); k <- k * dim^(-1/2) after the rotation
  per head:   S <- decay_h S + k v^T;   o = S^T q
  out = W_o (o / rms(o over the head's vdim) * silu(W_g h))          (the unit RMS has no weight)

S (fp32, [heads, dim, vdim]) is the sequence's state; it starts at zero. The
four projections of h run as one product (their matrices stacked at bind time).

Without a rotation nothing stands between the projections and the recurrence, so
recurrence, norm and gate run as one launch in a decode step and as chunks side
by side in a bfloat16 prompt step (`csrc/gated_memory.cu`, the kind with a fixed
decay a head).

Parameters: hidden_size, heads, dim, vdim, decay (one per head, not negative),
eps, rot (None or the parameters of a `rotary` position part), output ("act", the
default: rows in the run's activation type, or "fp32": unrounded, for a norm that
follows), and the tensors' names: q, k, v, g, o.
"""
from __future__ import annotations

import math
from typing import Mapping

import torch

from ..config.keys import ConfigError
from ..config.spec import PartSpec
from ..ops import kernels
from .base import CacheView, Mixer, StateRequest, TensorSpec, build_part, register_mixer


class Retention(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        g = lambda k: int(spec[k])
        self.D, self.H, self.dim, self.vd = g("hidden_size"), g("heads"), g("dim"), g("vdim")
        self.eps = float(spec["eps"])
        self.decay = [float(x) for x in spec["decay"]]
        self.names = {k: str(spec[k]) for k in ("q", "k", "v", "g", "o")}
        self.out_dtype = torch.float32 if str(spec.get("output", "act")) == "fp32" else None
        if len(self.decay) != self.H:
            raise ConfigError(f"retention: {len(self.decay)} decays for {self.H} heads")
        if any(not 0.0 <= x < math.inf for x in self.decay):
            raise ConfigError("retention: a decay is negative or not a number")
        if self.dim > 512 or self.vd > 512 and spec.get("rot") is None:
            raise ConfigError(f"retention: keys of {self.dim} values exceed the 512 that the recurrence kernel stages")
        rot = spec.get("rot")
        self.position = build_part("position", PartSpec("rotary", dict(rot))) if rot else None
        if self.position is not None and self.position.dims > self.dim:
            raise ConfigError(f"retention: {self.position.dims} rotated dims exceed the head's {self.dim}")

    def tensor_specs(self) -> list[TensorSpec]:
        n, H, D = self.names, self.H, self.D
        return [TensorSpec(n["q"], (H * self.dim, D)), TensorSpec(n["k"], (H * self.dim, D)),
                TensorSpec(n["v"], (H * self.vd, D)), TensorSpec(n["g"], (H * self.vd, D)),
                TensorSpec(n["o"], (D, H * self.vd))]

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        n = self.names
        self.at: dict[str, int] = {}
        parts, row = [], 0
        for k in ("q", "k", "v", "g"):
            self.at[k] = row
            parts.append(tensors[n[k]])
            row += tensors[n[k]].shape[0]
            # without a rotation every piece starts at a multiple of 8 rows of the stacked matrix; the last always ends at one
            if row % 8 and (self.position is None or k == "g"):
                parts.append(torch.zeros((8 - row % 8, self.D), dtype=parts[0].dtype, device=parts[0].device))
                row += 8 - row % 8
        self.w_all = torch.cat(parts, dim=0).contiguous()
        self.w_o = tensors[n["o"]]
        dev = self.w_o.device
        self.decay_t = torch.tensor(self.decay, dtype=torch.float32, device=dev)
        # a decay of zero has no logarithm: 2^-1e30 is zero all the same
        logs = [math.log2(x) if x > 0.0 else -1e30 for x in self.decay]
        self.decay_logs = torch.tensor(self.decay + logs, dtype=torch.float32, device=dev)
        self.ones = torch.ones((self.vd if self.position is not None else self.H * self.vd,), dtype=torch.float32, device=dev)
        self.cos = self.sin = None
        self.rot, self.interleaved = 0, False
        if self.position is not None:
            self.position.prepare(runtime)
            self.cos, self.sin, self.rot = self.position.fused_tables()
            self.interleaved = self.position.interleaved

    def streamed_tensors(self) -> list:
        return [self.w_all, self.w_o]

    def state_request(self):
        return {"S": StateRequest((self.H, self.dim, self.vd), torch.float32)}

    def forward(self, h: torch.Tensor, ctx, cache: CacheView) -> torch.Tensor:
        H, dim, vd = self.H, self.dim, self.vd
        p = kernels.linear(h, self.w_all)
        if self.position is None:
            out = torch.empty((p.shape[0], H * vd), dtype=p.dtype, device=p.device)
            kernels.gated_memory("fixed", p, self.at, None, self.decay_logs, self.ones, float(dim) ** -0.5, cache.state, out, ctx, H, dim,
                                 vd, self.eps)
            return kernels.linear(out, self.w_o, out_dtype=self.out_dtype)
        nq = H * dim
        qn, kn = kernels.retention_prep(p, 0, nq, H, dim, self.cos, self.sin, self.rot, self.interleaved,
                                        float(dim) ** -0.5, ctx)
        o = kernels.retention_scan(qn, kn, p, 2 * nq, self.decay_t, cache.state["S"], ctx, H, dim, vd)
        out = kernels.gated_rmsnorm(o, p[:, 2 * nq + H * vd: 2 * nq + 2 * H * vd], self.ones, H, vd, self.eps)
        return kernels.linear(out, self.w_o, out_dtype=self.out_dtype)


register_mixer("retention", Retention)
