"""Softmax attention over one latent vector per position: every head's keys and
values are linear maps of the latent, and one rotated key part is shared by all
heads. Only the latent and that part are cached.

With h the mixer's input, H heads, per head `dim` unrotated and `rot_dim`
rotated query/key dimensions, values of `vdim`, a latent of `kv_rank`:

  q = W_q h, or, with a latent of the queries' own of `q_rank`, q = W_q rms_norm(W_dq h) * w_dq
                                 per head [dim unrotated | rot_dim rotated]
  d = W_dkv h                    kv_rank + rot_dim outputs
  c = rms_norm(d[:kv_rank]) * w  (plain weight)      k_r = d[kv_rank:]     (not normed)
  q_r (every head) and k_r are rotated (the position part's pairing, tables and scaling)
  per head:  k_u = W_uk c,  v = W_uv c,  score = (q_u . k_u + q_r . k_r) * scale
  causal softmax (within `window` when given), W_o on the concatenated heads
  with `gate` (a tensor name): head h's output is multiplied by sigmoid(W_g h)_h first; W_g [H, hidden] reads the
  same input as the projections; with gate_kind "value" W_g is [H * vdim, hidden] and every value has a gate of its own

The maps move to the query side (`csrc/latent_attn.cu`): q_a = W_uk^T q_u per
head, the cache row of a position is [c | k_r] for ONE kv head, the library's
attention kernels run with that row as key and as value, and W_uv maps the
first kv_rank columns of their output to the head's values. A run that reads
another run's cache (`cache_from` in the schedule) has no W_dkv: it brings its
own queries, W_uk, W_uv and W_o.

Parameters: hidden_size, heads, dim, rot_dim, vdim, kv_rank, eps, scale, window,
rot (None or the parameters of a `rotary` position part), own_kv (False for a
run that reads another's cache), gate (None, or the name of the output gate's
matrix), gate_kind ("head" | "value"), q_rank (None: queries come from h; an
integer, or -1: what the checkpoint's tensors have), pad_heads (False), output
("act", the default: rows in the run's activation type, or "fp32": unrounded, for
a norm that follows), and the tensors' names: q, dkv, dkv_norm, uk, uv, o; dq and
dq_norm with q_rank.

Cache rows are padded with zeros to a multiple of 8 values (the attention
kernels' 16-byte loads), or, with `pad_heads`, to the 64 or 128 that the
tensor-core kernels take where they fit.
"""
from __future__ import annotations

from typing import Mapping, Optional

import torch

from ..config.keys import ConfigError
from ..config.spec import PartSpec
from ..ops import attention_dispatch, kernels
from .base import CacheView, KVRequest, Mixer, TensorSpec, build_part, register_mixer


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class LatentAttention(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        g = lambda k: int(spec[k])
        self.D, self.H, self.dim, self.rd, self.vd, self.r = (g("hidden_size"), g("heads"), g("dim"), g("rot_dim"),
                                                              g("vdim"), g("kv_rank"))
        self.eps, self.scale = float(spec["eps"]), float(spec["scale"])
        self.window: Optional[int] = spec.get("window")
        self.own_kv = bool(spec.get("own_kv", True))
        self.names = {k: str(spec[k]) for k in ("q", "dkv", "dkv_norm", "uk", "uv", "o")}
        self.gate_name: Optional[str] = spec.get("gate")
        self.gate_kind = str(spec.get("gate_kind", "head"))
        if self.gate_kind not in ("head", "value"):
            raise ConfigError(f"latent_attention: gate_kind {self.gate_kind!r} is neither 'head' nor 'value'")
        self.n_gates = 0 if not self.gate_name else self.H if self.gate_kind == "head" else self.H * self.vd
        self.q_rank: Optional[int] = None if spec.get("q_rank") is None else int(spec["q_rank"])
        if self.q_rank is not None:
            self.names.update({k: str(spec[k]) for k in ("dq", "dq_norm")})
        self.out_dtype = torch.float32 if str(spec.get("output", "act")) == "fp32" else None
        n = self.r + self.rd
        self.HDp = 64 if spec.get("pad_heads") and n <= 64 else 128 if spec.get("pad_heads") and n <= 128 else _pad8(n)
        if self.HDp > kernels.MAX_HEAD_DIM:
            raise ConfigError(f"latent_attention: a cache row of {self.r} + {self.rd} values exceeds {kernels.MAX_HEAD_DIM}")
        if self.window is not None and self.window < 1:
            raise ConfigError(f"latent_attention: window {self.window} must be positive")
        rot = spec.get("rot")
        self.position = None
        if rot and self.rd:
            self.position = build_part("position", PartSpec("rotary", dict(rot)))
            if self.position.dims > self.rd:
                raise ConfigError(f"latent_attention: {self.position.dims} rotated dims exceed the rotated part of {self.rd}")

    def tensor_specs(self) -> list[TensorSpec]:
        n, H, D, r = self.names, self.H, self.D, self.r
        specs = [TensorSpec(n["q"], (H * (self.dim + self.rd), D if self.q_rank is None else self.q_rank), free_size=64),
                 TensorSpec(n["uk"], (H * self.dim, r)), TensorSpec(n["uv"], (H * self.vd, r)),
                 TensorSpec(n["o"], (D, H * self.vd))]
        if self.gate_name:
            specs.append(TensorSpec(self.gate_name, (self.n_gates, D)))
        if self.q_rank is not None:
            specs += [TensorSpec(n["dq"], (self.q_rank, D), free_size=64),
                      TensorSpec(n["dq_norm"], (self.q_rank,), role="gain", init="gain", std=0.1, free_size=64)]
        if self.own_kv:
            specs += [TensorSpec(n["dkv"], (r + self.rd, D)),
                      TensorSpec(n["dkv_norm"], (r,), role="gain", init="gain", std=0.1)]
        return specs

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        n = self.names
        # the first product's rows: the queries (or their latent), the down-projection, the gate's logits
        wq = tensors[n["q"]] if self.q_rank is None else tensors[n["dq"]]
        self.n_q = wq.shape[0]
        self.w_uq = self.dq_gain = None
        if self.q_rank is not None:
            self.w_uq, self.dq_gain = tensors[n["q"]], tensors[n["dq_norm"]]
            if self.w_uq.shape[1] != self.n_q or self.dq_gain.numel() != self.n_q:
                raise ConfigError(f"latent_attention: {n['dq']}, {n['dq_norm']} and {n['q']} do not agree on the queries' latent")
        parts = [wq]
        if self.own_kv:
            parts.append(tensors[n["dkv"]])
        self.norm_w = tensors[n["dkv_norm"]] if self.own_kv else None
        rows = sum(t.shape[0] for t in parts)
        self.gate_off = rows                     # the gate's logits follow the projections in the same product
        if self.gate_name:
            parts.append(tensors[self.gate_name])
            rows += self.n_gates
        if len(parts) > 1 and rows % 8:
            parts.append(torch.zeros((8 - rows % 8, self.D), dtype=wq.dtype, device=wq.device))
        self.w_in = torch.cat(parts, dim=0).contiguous() if len(parts) > 1 else wq
        # W_uk per head, transposed: q_a[r] = sum_i W_uk[h, i, r] q_u[i]
        self.w_ukT = tensors[n["uk"]].view(self.H, self.dim, self.r).transpose(1, 2).contiguous()
        self.w_uv = tensors[n["uv"]].view(self.H, self.vd, self.r).contiguous()
        self.w_o = tensors[n["o"]]
        self.cos = self.sin = None
        self.rot, self.interleaved = 0, False
        if self.position is not None:
            self.position.prepare(runtime)
            self.cos, self.sin, self.rot = self.position.fused_tables()
            self.interleaved = self.position.interleaved
        self.runtime = runtime

    def streamed_tensors(self) -> list:
        return [t for t in (self.w_in, self.w_uq, self.w_ukT, self.w_uv, self.w_o) if t is not None]

    def kv_request(self) -> KVRequest:
        return KVRequest(1, self.HDp, self.window, values=False)

    def forward(self, h: torch.Tensor, ctx, cache: CacheView) -> torch.Tensor:
        if cache.writes != self.own_kv:
            raise ConfigError("latent_attention: a layer with a down-projection keeps its own cache, one without reads another's")
        H, HDp, r = self.H, self.HDp, self.r
        T = h.shape[0]
        pages = ctx.pages[cache.group]
        p = kernels.linear(h, self.w_in)
        q = torch.empty((T, H * HDp), dtype=p.dtype, device=p.device)
        qr = p if self.w_uq is None else kernels.linear(kernels.rms_rows(p, self.n_q, self.dq_gain, self.eps), self.w_uq)
        kernels.latent_prep(qr, 0, p if self.own_kv else None, self.n_q, q, H, self.dim, self.rd, r, HDp,
                            self.norm_w, self.eps, self.cos, self.sin, self.rot, self.interleaved, ctx, pages,
                            cache.k if self.own_kv else None)
        kernels.head_linear(qr, self.dim + self.rd, 0, self.w_ukT, q, HDp, 0)
        lat = torch.empty((T, H * HDp), dtype=p.dtype, device=p.device)
        if ctx.is_decode:
            scratch = self.runtime.attn_scratch(ctx.B, H, HDp, ctx.decode_splits)
            # the tensor-core decode kernel takes up to 16 query heads a kv head: more heads go in groups of 16
            G = 16 if (H > 16 and attention_dispatch.USE_TC_MASKED and kernels.attn_decode_tc_supported(p.dtype, 16, 1, HDp)
                       and attention_dispatch._tc_fits(16, 1, ctx.decode_splits)) else H
            for h0 in range(0, H, G):
                n = min(G, H - h0)
                cols = slice(h0 * HDp, (h0 + n) * HDp)
                attention_dispatch.decode_masked(q[:, cols] if n < H else q, lat[:, cols] if n < H else lat, ctx, n, 1, HDp,
                                                 HDp, cache.k, cache.k, pages, self.window or 0, 0, self.scale, scratch)
        else:
            attention_dispatch.prefill_masked(q, lat, ctx, H, 1, HDp, HDp, cache.k, cache.k, pages, self.window or 0, 0,
                                              self.scale)
        v = torch.empty((T, H * self.vd), dtype=p.dtype, device=p.device)
        # the gate rides on the value product's accumulators
        kernels.head_linear(lat, HDp, 0, self.w_uv, v, self.vd, 0,
                            gate=p[:, self.gate_off: self.gate_off + self.n_gates] if self.gate_name else None,
                            gate_cols=self.gate_kind == "value")
        return kernels.linear(v, self.w_o, out_dtype=self.out_dtype)


register_mixer("latent_attention", LatentAttention)
