"""Chooses the attention kernel of a step.

The tensor-core kernel takes bfloat16 with the head sizes it was built for;
everything else (the whole 32-bit path, other head sizes) runs the general
kernel. Both read the same paged cache and give the same result up to
rounding.
"""
from __future__ import annotations

import os

import torch

from . import kernels


# Switch for the tcgen05 prompt attention (tests compare it with the mma.sync kernel).
USE_TCGEN05_PREFILL = os.environ.get("MYNAH_TCGEN05_ATTN", "1") != "0"


def prefill(qkv: torch.Tensor, out: torch.Tensor, ctx, H: int, KV: int, HD: int,
            k_cache: torch.Tensor, v_cache: torch.Tensor, pages, window: int) -> None:
    if USE_TCGEN05_PREFILL and kernels.attn_prefill_tcgen05_supported(qkv.dtype, H, KV, HD):
        kernels.attn_prefill_tcgen05(qkv, out, ctx.B, ctx.max_q_len, H, KV, HD, k_cache, v_cache,
                                     ctx.cu_q, ctx.kv_len, pages, window, ctx.status)
        return
    if kernels.attn_prefill_tc_supported(qkv.dtype, H, KV, HD):
        kernels.attn_prefill_tc(qkv, out, ctx.B, ctx.max_q_len, H, KV, HD, k_cache, v_cache,
                                ctx.cu_q, ctx.kv_len, pages, window, ctx.status)
        return
    kernels.attn_prefill_generic(qkv, out, ctx.B, ctx.max_q_len, H, KV, HD, k_cache, v_cache,
                                 ctx.cu_q, ctx.kv_len, pages, window, ctx.status)


# The one-launch decode attention (norm, rotation, cache write, pages, merge) saves two launches but repeats
# the query's preparation in every page's CTA, so it pays while a step has few CTAs. Both routes give a
# sequence the same bits, so the choice may depend on the batch. 0 switches it off.
FUSED_DECODE_MAX_CTAS = int(os.environ.get("MYNAH_FUSED_ATTN_MAX_CTAS", "1100"))
# Floats of shared memory that the merge of a (sequence, kv head) has for its pages' weights.
_MERGE_FLOATS = 2048


def _tc_fits(H: int, KV: int, n_splits: int) -> bool:
    return (H // KV) * n_splits <= _MERGE_FLOATS


# Larger steps can still let the pages' kernel prepare the queries and write the new key and value itself (no
# rotation/cache-write launch before it) and merge with a launch of its own. 1: do so.
FUSED_PREP_LARGE = os.environ.get("MYNAH_FUSED_ATTN_PREP", "0") == "1"


def decode_fused_ok(dtype: torch.dtype, H: int, KV: int, HD: int, rotary_dim: int, cos, B: int, n_splits: int) -> bool:
    """Whether the one-launch decode attention takes this layer in this step: the tensor-core sizes, a rotation
    of the whole head or none, and few enough CTAs."""
    if not kernels.attn_decode_tc_supported(dtype, H, KV, HD):
        return False
    if B * KV * n_splits > FUSED_DECODE_MAX_CTAS and not FUSED_PREP_LARGE:
        return False
    return _tc_fits(H, KV, n_splits) and (cos is None or rotary_dim == HD)


def decode_fused_merges(B: int, KV: int, n_splits: int) -> bool:
    """Whether the one-launch form also merges (small steps), or leaves the merge to a launch of its own."""
    return B * KV * n_splits <= FUSED_DECODE_MAX_CTAS


# Whether the pages' kernel of the tensor-core decode attention also merges (the CTA that finishes a sequence's
# kv head last), instead of a merge launch of its own with a CTA per head. The bits are the same; the launch of its
# own measured faster (batch 8: 1.37 against 1.48 ms a step; batch 64: 3.92 against 4.60), so this is off.
MERGE_IN_PAGES_KERNEL = os.environ.get("MYNAH_ATTN_MERGE_IN_PAGES", "0") == "1"


def decode(qkv: torch.Tensor, out: torch.Tensor, ctx, H: int, KV: int, HD: int, k_cache: torch.Tensor,
           v_cache: torch.Tensor, pages, window: int, scratch: torch.Tensor, counters=None) -> None:
    """One query per sequence. Both kernels split a sequence page by page and
    combine in page order, so either gives a sequence the same bits whatever
    the batch."""
    if kernels.attn_decode_tc_supported(qkv.dtype, H, KV, HD) and _tc_fits(H, KV, ctx.decode_splits):
        kernels.attn_decode_tc(qkv, out, ctx.B, H, KV, HD, k_cache, v_cache, ctx.kv_len, pages, window,
                               ctx.decode_splits, scratch, ctx.status,
                               counters if MERGE_IN_PAGES_KERNEL else None)
    else:
        kernels.attn_decode(qkv, out, ctx.B, H, KV, HD, k_cache, v_cache, ctx.kv_len, pages, window,
                            ctx.decode_splits, scratch, ctx.status)


# Switch for the tensor-core kernels under mixers with a chunk mask or a scale of their own (tests compare them with
# the general kernels).
USE_TC_MASKED = os.environ.get("MYNAH_TC_MASKED_ATTN", "1") != "0"


def prefill_masked(q: torch.Tensor, out: torch.Tensor, ctx, H: int, KV: int, HD: int, VD: int, k_cache, v_cache, pages,
                   window: int, chunk: int, scale: float) -> None:
    """Prompt attention for mixers with a chunk mask, a score scale of their own or value heads of another width:
    the tcgen05 kernel where it takes the sizes (bfloat16, keys and values of one width, 64 or 128, a positive
    scale), else the general kernel. Both give the same result up to rounding."""
    if (USE_TC_MASKED and USE_TCGEN05_PREFILL and HD == VD and scale > 0.0 and kernels.attn_prefill_tcgen05_supported(q.dtype, H, KV, HD)):
        kernels.attn_prefill_tcgen05_masked(q, out, ctx, H, KV, HD, k_cache, v_cache, pages, window, chunk, scale)
        return
    kernels.attn_prefill_general(q, out, ctx, H, KV, HD, VD, k_cache, v_cache, pages, window, chunk, scale)


def decode_masked(q: torch.Tensor, out: torch.Tensor, ctx, H: int, KV: int, HD: int, VD: int, k_cache, v_cache, pages,
                  window: int, chunk: int, scale: float, scratch: torch.Tensor) -> None:
    """The same choice for a decode step (the tensor-core kernel takes a window or a chunk, not both)."""
    if (USE_TC_MASKED and HD == VD and not (window and chunk) and kernels.attn_decode_tc_supported(q.dtype, H, KV, HD)
            and _tc_fits(H, KV, ctx.decode_splits)):
        kernels.attn_decode_tc_masked(q, out, ctx, H, KV, HD, k_cache, v_cache, pages, window, chunk, scale, scratch)
        return
    kernels.attn_decode_general(q, out, ctx, H, KV, HD, VD, k_cache, v_cache, pages, window, chunk, scale, scratch)


def _tc_capped_fits(HD: int, VD: int, scale: float, softcap: float, vdo: int) -> bool:
    """Whether the tensor-core kernels take these heads: widths of 64 or 128 (one width for both under a cap), output heads
    of whole 16-byte pieces."""
    return USE_TC_MASKED and scale > 0.0 and VD in (64, 128) and (VD == HD or not softcap) and vdo % 8 == 0


def prefill_capped(q: torch.Tensor, out: torch.Tensor, ctx, H: int, KV: int, HD: int, VD: int, k_cache, v_cache, pages,
                   window: int, scale: float, softcap: float, keep_first: int, vdiv: int, null_key: bool = False,
                   out_scale: float = 1.0, vdo=None, sink=None) -> None:
    """Prompt attention for mixers whose scores are capped, whose window keeps a sequence's first tokens, whose key heads
    share value heads (`vdiv` key heads a value head), whose softmax holds one more term without a value, of score 0
    (`null_key`) or of a score of its own for every query head (`sink`), whose output carries a factor, or whose output heads are narrower (`vdo` columns) than the stored value
    heads. Without any of these it is `prefill_masked`; the tcgen05 kernel takes bfloat16 heads of 64 or 128, the general
    kernel the rest."""
    vdo = VD if vdo is None else int(vdo)
    plain = not null_key and sink is None and out_scale == 1.0 and vdo == VD
    if plain and not softcap and not keep_first and vdiv == 1 and out.is_contiguous():
        prefill_masked(q, out, ctx, H, KV, HD, VD, k_cache, v_cache, pages, window, 0, scale)
        return
    if (USE_TCGEN05_PREFILL and _tc_capped_fits(HD, VD, scale, softcap, vdo)
            and kernels.attn_prefill_tcgen05_supported(q.dtype, H, KV, HD)):
        kernels.attn_prefill_tcgen05_capped(q, out, ctx, H, KV, HD, k_cache, v_cache, pages, window, scale, softcap,
                                            keep_first, vdiv, VD, null_key, out_scale, vdo, sink)
        return
    kernels.attn_prefill_capped(q, out, ctx, H, KV, HD, VD, k_cache, v_cache, pages, window, scale, softcap, keep_first, vdiv,
                                null_key, out_scale, vdo, sink)


def decode_capped(q: torch.Tensor, out: torch.Tensor, ctx, H: int, KV: int, HD: int, VD: int, k_cache, v_cache, pages,
                  window: int, scale: float, softcap: float, keep_first: int, vdiv: int, scratch: torch.Tensor,
                  null_key: bool = False, out_scale: float = 1.0, vdo=None, sink=None) -> None:
    """The same choice for a decode step."""
    vdo = VD if vdo is None else int(vdo)
    plain = not null_key and sink is None and out_scale == 1.0 and vdo == VD
    if plain and not softcap and not keep_first and vdiv == 1 and out.is_contiguous():
        decode_masked(q, out, ctx, H, KV, HD, VD, k_cache, v_cache, pages, window, 0, scale, scratch)
        return
    if (_tc_capped_fits(HD, VD, scale, softcap, vdo) and kernels.attn_decode_tc_supported(q.dtype, H, KV, HD)
            and _tc_fits(H, KV, ctx.decode_splits)):
        kernels.attn_decode_tc_capped(q, out, ctx, H, KV, HD, k_cache, v_cache, pages, window, scale, softcap, keep_first,
                                      vdiv, scratch, VD, null_key, out_scale, vdo, sink)
        return
    kernels.attn_decode_capped(q, out, ctx, H, KV, HD, VD, k_cache, v_cache, pages, window, scale, softcap, keep_first, vdiv,
                               scratch, null_key, out_scale, vdo, sink)
