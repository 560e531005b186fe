"""Token embedding and output head.

Embedding: x = E[token], no scaling by sqrt(hidden) (mynah-slm
src/arch_qwen3.c:186); a design that multiplies its embedding by a constant
gives `scale` (the product is fp32), and one that multiplies its logits by a
constant gives the head `logit_scale`; one that caps its logits gives
`logit_softcap` c: c tanh(logits / c). Head: logits = Head . h in fp32, where Head is the
embedding matrix when the configuration ties them and `lm_head.weight`
otherwise; the configuration decides, not the presence of the tensor
(docs/qwen3-arch.md:91-113: the official checkpoint ships a duplicate
`lm_head.weight` although it is tied).
"""
from __future__ import annotations

from typing import Mapping, Optional

import torch

from ..ops import kernels
from .base import Embedding, Head, Part, StateRequest, TensorSpec, register_embedding, register_head


class TokenEmbedding(Embedding):
    def __init__(self, spec):
        super().__init__(spec)
        self.name = str(spec["name"])
        self.V, self.D = int(spec["vocab_size"]), int(spec["dim"])
        self.scale = float(spec.get("scale", 1.0))
        self.table: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        return [TensorSpec(self.name, (self.V, self.D))]

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        self.table = tensors[self.name]

    def forward(self, tokens: torch.Tensor) -> torch.Tensor:
        return kernels.embed_gather(self.table, tokens, scale=self.scale)


class LinearHead(Head):
    def __init__(self, spec, embedding):
        super().__init__(spec)
        self.tied = bool(spec["tied"])
        self.name = str(spec["name"])
        self.V, self.D = int(spec["vocab_size"]), int(spec["dim"])
        self.embedding = embedding
        self.logit_scale = float(spec.get("logit_scale", 1.0))
        self.logit_softcap = float(spec.get("logit_softcap") or 0.0)
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        # tied: a stored copy is tolerated and left unread
        return [TensorSpec(self.name, (self.V, self.D), ignorable=self.tied)]

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        if self.tied and getattr(self.embedding, "table", None) is None:
            from ..config.keys import ConfigError
            raise ConfigError("linear_head: a tied head needs an embedding part that keeps its matrix as `table`")
        self.weight = self.embedding.table if self.tied else tensors[self.name]

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        logits = kernels.linear(h, self.weight, out_dtype=torch.float32)
        if self.logit_scale != 1.0:
            logits = kernels.scale_(logits, self.logit_scale)
        return kernels.softcap_(logits, self.logit_softcap) if self.logit_softcap else logits


register_embedding("token_embedding", TokenEmbedding)
register_head("linear_head", LinearHead)


class TokenPositionEmbedding(Embedding):
    """x = E[token] + P[position]: a learned vector per absolute position, added unscaled to the token's.
    Parameters: name, position_name, vocab_size, dim, max_positions. It reads the rows' positions, so the
    engine hands it the step's context."""
    needs_context = True

    def __init__(self, spec):
        super().__init__(spec)
        self.name, self.pos_name = str(spec["name"]), str(spec["position_name"])
        self.V, self.D, self.P = int(spec["vocab_size"]), int(spec["dim"]), int(spec["max_positions"])
        self.table: Optional[torch.Tensor] = None
        self.pos_table: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        return [TensorSpec(self.name, (self.V, self.D)), TensorSpec(self.pos_name, (self.P, self.D))]

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        self.table, self.pos_table = tensors[self.name], tensors[self.pos_name]

    def forward(self, tokens: torch.Tensor, ctx) -> torch.Tensor:
        return kernels.embed_positions(self.table, self.pos_table, tokens, ctx.tok_pos, ctx.status)


register_embedding("token_position_embedding", TokenPositionEmbedding)


class TokenPairEmbedding(Embedding):
    """x = E[token] + P[row]: a second table looked up by the token and the one before it, row = (token before * mul_prev
    + token * mul_cur) mod buckets; a sequence's first token takes the table's last row (number `buckets`). Every
    sequence's last token is kept as its state, so that a piece of a prompt or a decoded token finds the one before it.
    Parameters: name, pair_name, vocab_size, dim, buckets, mul_prev, mul_cur."""
    needs_context = True

    def __init__(self, spec):
        super().__init__(spec)
        self.name, self.pair_name = str(spec["name"]), str(spec["pair_name"])
        self.V, self.D, self.buckets = int(spec["vocab_size"]), int(spec["dim"]), int(spec["buckets"])
        # only the multipliers' remainders matter
        self.mul_prev, self.mul_cur = int(spec["mul_prev"]) % self.buckets, int(spec["mul_cur"]) % self.buckets
        self.table: Optional[torch.Tensor] = None
        self.pairs: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        return [TensorSpec(self.name, (self.V, self.D)), TensorSpec(self.pair_name, (self.buckets + 1, self.D))]

    def bind(self, tensors: Mapping[str, torch.Tensor], runtime) -> None:
        self.table, self.pairs = tensors[self.name], tensors[self.pair_name]

    def state_request(self):
        return StateRequest((), torch.int32)

    def forward(self, tokens: torch.Tensor, ctx, state: torch.Tensor) -> torch.Tensor:
        return kernels.embed_pairs(self.table, self.pairs, state, ctx, self.mul_prev, self.mul_cur)


register_embedding("token_pair_embedding", TokenPairEmbedding)


class StreamVectors(Part):
    """Learned vectors [count, dim] that the schedule adds to every row of the residual stream before chosen runs
    (`ScheduleEntry.add_vector`); kept in fp32, like the stream. Parameters: name, count, dim."""

    def __init__(self, spec):
        super().__init__(spec)
        self.name, self.count, self.dim = str(spec["name"]), int(spec["count"]), int(spec["dim"])
        self.rows = None

    def tensor_specs(self) -> list[TensorSpec]:
        return [TensorSpec(self.name, (self.count, self.dim), role="gain", init="normal", std=0.1)]

    def bind(self, tensors, runtime) -> None:
        self.rows = tensors[self.name].to(torch.float32).contiguous()
