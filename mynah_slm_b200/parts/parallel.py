"""Two mixers side by side that read the same input, in one of two forms.

With `out_norms`, each output is RMS-normed over the model width with a plain gain of its own, and the result is
their weighted sum:

  out = weight * (a / rms(a) * g_a + b / rms(b) * g_b),   a = left(h),  b = right(h)

The sum and both norms are fp32 (`csrc/norm_post.cu`); the branches hand over fp32 rows.

With `scales`, the result is scale_a * a + scale_b * b. Both branches must then be mixers that offer the two halves of
their work (`shares_products`: a product of h, the heads, a product of the heads' rows): the two products of h run as
one, the heads of both branches lie side by side in the rows of one matrix, each already times its scale (which a
branch applies in fp32, before it rounds its rows), and one product makes the sum.
 Each branch is a mixer of any registered kind, built from its own
`PartSpec`. At most one branch keeps keys and values (a run of a layer has one
place in a storage group); the branches' fixed-size states are asked for side
by side, branch i's under the name "i".

Parameters: hidden_size, branches (two PartSpecs), and either eps, weight and out_norms (the two gains' tensor names)
or scales (two factors).
"""
from __future__ import annotations

from typing import Mapping

import torch

from ..config.keys import ConfigError
from ..config.spec import PartSpec
from ..ops import kernels
from .base import CacheView, Mixer, TensorSpec, build_part, register_mixer


class ParallelMixers(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        self.D = int(spec["hidden_size"])
        self.eps = float(spec.get("eps", 0.0))
        self.weight = float(spec.get("weight", 0.5))
        self.scales = tuple(float(x) for x in spec["scales"]) if spec.get("scales") is not None else None
        branches = tuple(spec["branches"])
        self.gain_names = tuple(str(n) for n in spec.get("out_norms") or ())
        if len(branches) != 2 or (self.scales is None) != (len(self.gain_names) == 2) or len(self.scales or (0, 0)) != 2:
            raise ConfigError("parallel_mixers: exactly two branches, each with the gain of its output's norm or with a factor")
        self.branches = [build_part("mixer", b) for b in branches]
        if self.scales is not None:
            for b, x in zip(self.branches, self.scales):
                if not getattr(b, "shares_products", False):
                    raise ConfigError(f"parallel_mixers: {b.spec.kind!r} does not offer the halves of its work, which a sum with factors needs")
                b.out_scale = x
        if sum(b.kv_request() is not None for b in self.branches) > 1:
            raise ConfigError("parallel_mixers: only one branch may keep keys and values")

    def tensor_specs(self) -> list[TensorSpec]:
        specs = [ts for b in self.branches for ts in b.tensor_specs()]
        return specs + [TensorSpec(n, (self.D,), role="gain", init="gain", std=0.1) for n in self.gain_names]

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        for b in self.branches:
            b.bind({ts.name: tensors[ts.name] for ts in b.tensor_specs() if ts.name in tensors}, runtime)
        if self.scales is not None:
            # the branches' matrices as one: rows side by side under h, columns side by side over the heads' rows, every
            # branch's columns from a multiple of 8 on
            self.in_cols, self.out_at = [], []
            ins, outs, row, col = [], [], 0, 0
            for b in self.branches:
                w, o = b.in_weight, b.out_weight
                pad_r, pad_c = -w.shape[0] % 8, -o.shape[1] % 8
                ins += [w] + ([torch.zeros((pad_r, self.D), dtype=w.dtype, device=w.device)] if pad_r else [])
                outs += [o] + ([torch.zeros((self.D, pad_c), dtype=o.dtype, device=o.device)] if pad_c else [])
                self.in_cols.append((row, row + w.shape[0]))
                self.out_at.append((col, col + o.shape[1]))
                row, col = row + w.shape[0] + pad_r, col + o.shape[1] + pad_c
                b.in_weight = b.out_weight = None              # they live on in the joint matrices
            self.w_in, self.w_out = torch.cat(ins, dim=0).contiguous(), torch.cat(outs, dim=1).contiguous()
            self.out_padded = sum(b - a for a, b in self.out_at) != col
            return
        g0 = tensors[self.gain_names[0]]
        self.gains = (g0.contiguous(), tensors[self.gain_names[1]].to(g0.dtype).contiguous())

    def streamed_tensors(self) -> list:
        if self.scales is not None:
            return [self.w_in, self.w_out]
        return [t for b in self.branches for t in b.streamed_tensors()]

    def kv_request(self):
        for b in self.branches:
            if b.kv_request() is not None:
                return b.kv_request()
        return None

    def state_request(self):
        req = {str(i): b.state_request() for i, b in enumerate(self.branches) if b.state_request() is not None}
        return req or None

    def _view(self, i: int, cache: CacheView) -> CacheView:
        state = cache.state.get(str(i)) if cache.state is not None else None
        keeps = self.branches[i].kv_request() is not None
        return CacheView(group=cache.group, k=cache.k if keeps else None, v=cache.v if keeps else None, writes=cache.writes,
                         state=state)

    def forward(self, h: torch.Tensor, ctx, cache: CacheView) -> torch.Tensor:
        if self.scales is not None:
            p = kernels.linear(h, self.w_in)
            make = torch.zeros if self.out_padded else torch.empty
            rows = make((p.shape[0], self.w_out.shape[1]), dtype=p.dtype, device=p.device)
            for i, b in enumerate(self.branches):
                b.heads(p[:, self.in_cols[i][0]: self.in_cols[i][1]], rows[:, self.out_at[i][0]: self.out_at[i][1]], ctx,
                        self._view(i, cache))
            return kernels.linear(rows, self.w_out)
        outs = []
        for i, b in enumerate(self.branches):
            y = b.forward(h, ctx, self._view(i, cache))
            if y.dtype != torch.float32:
                raise ConfigError("parallel_mixers: a branch must hand over fp32 rows")
            outs.append(y)
        return kernels.rms_pair_mean(outs[0], outs[1], self.gains[0], self.gains[1], self.eps, self.weight)


register_mixer("parallel_mixers", ParallelMixers)
