"""Chooses the attention kernels for a step.

float32 (the true 32-bit path): the CUDA-core kernel serves every row.
bfloat16: rows with one new token go to the tensor-core decode kernel (context split across
blocks), rows with more go to a prefill kernel -- the tcgen05 one for head sizes 64 and 128, the
mma.sync one for the other multiples of 16 up to 128; head sizes beyond those kernels fall back to
the CUDA-core kernel, which takes every size up to 256.  ``set_backend("simt")`` forces the CUDA-core
kernel everywhere (used by tests to compare the two)."""
from __future__ import annotations

import torch

from . import ops

_backend = "auto"
_prefill_backend = "tcgen05"


def set_prefill_backend(name: str) -> None:
    global _prefill_backend
    if name not in ("tcgen05", "mma"):
        raise ValueError(name)
    _prefill_backend = name


def set_backend(name: str) -> None:
    global _backend
    if name not in ("auto", "simt"):
        raise ValueError(name)
    _backend = name


def _row_kinds(ctx) -> tuple:
    """(rows of one token, rows of more, tokens of those) of the step, or None where the host does not know the rows'
    lengths (a captured step).  Counted once a step, not once a layer: a step may hold hundreds of rows."""
    kinds = ctx.host.get("_row_kinds", False)
    if kinds is False:
        q_lens = ctx.host.get("q_len")
        kinds = None
        if q_lens is not None:
            long = [n for n in q_lens if n > 1]
            kinds = (len(q_lens) - len(long), len(long), sum(long))
        ctx.host["_row_kinds"] = kinds
    return kinds


def decode_only(ctx) -> bool:
    """Whether every row of the step has exactly one new token (known on the host)."""
    kinds = _row_kinds(ctx)
    return kinds is not None and kinds[1] == 0 and kinds[0] > 0


def rotates_in_decode(dtype, head_dim: int, ctx) -> bool:
    """Whether ``attention(..., rope=...)`` can rotate q and the new key itself and write the cache: a step of
    decoding rows only, on the tensor-core decode kernel, with a head size it rotates."""
    return (_backend == "auto" and dtype == torch.bfloat16 and head_dim <= 128 and head_dim % 32 == 0
            and decode_only(ctx))


def attention(qkv, ctx, cache, out, num_heads, num_kv_heads, head_dim, scale, window, rope=None, q_stride=None, mods=None,
              keep: int = 0):
    """``rope`` = (cos, sin): ``qkv`` is unrotated and the cache rows of the new tokens are unwritten; only
    where ``rotates_in_decode`` holds.  ``window``: None or 0 all earlier keys, w > 0 the last w positions, w < 0 the
    keys of the query's own block of -w positions.  ``keep``: beside a window or block, the first ``keep`` keys of the
    sequence stay in sight.  ``q_stride``: elements between the token rows of ``qkv`` (by
    default rows of a fused q|k|v projection).  ``mods`` (``ops.ScoreMods``): a cap on the scores, a bias or a slope by distance, a sink in
    the softmax; every kernel applies them (the tcgen05 kernel for portions in an instance of its own)."""
    if q_stride is None:
        q_stride = (num_heads + 2 * num_kv_heads) * head_dim
    args = (qkv, q_stride, cache.k, cache.v, ctx.block_tables[cache.group], ctx.row_q_start, ctx.row_q_len,
            ctx.row_ctx_len)
    fast = _backend == "auto" and qkv.dtype == torch.bfloat16 and head_dim <= 128
    window = int(window or 0)
    # the keys a single new token can reach, for the decode kernel's plan: a window or a block of positions bounds them
    keep = int(keep or 0) if window else 0              # (without a window every key is in sight already)
    reach = ctx.max_ctx_len if window == 0 else min(ctx.max_ctx_len, abs(window) + 64 + -(-keep // 64) * 64)
    if rope is not None:
        if mods is not None or keep:
            raise ValueError("rotation inside attention does not go together with score modifiers or kept keys")
        if not rotates_in_decode(qkv.dtype, head_dim, ctx):
            raise ValueError("rotation inside attention serves steps of decoding rows only (bfloat16, head sizes "
                             "in steps of 32 up to 128)")
        return ops.decode_attention(*args, out, num_heads, num_kv_heads, head_dim, cache.page_size, scale, window,
                                    max_ctx=ctx.max_ctx_len, rope=rope)
    if not fast:
        return ops.paged_attention(*args, ctx.num_tokens, out, num_heads, num_kv_heads, head_dim, cache.page_size,
                                   scale, window, mods=mods, keep=keep)
    kinds = _row_kinds(ctx)
    has_decode = kinds is None or kinds[0] > 0
    has_prefill = kinds is None or kinds[1] > 0
    min_q_len = 2
    if kinds is None and ctx.host.get("few_single_rows"):
        # row lengths unknown here (a captured step), but rows of one token are the exception among them: the
        # kernel for portions takes those too, and the launch of the decode kernel is saved
        has_decode, min_q_len = False, 1
    if has_decode:
        ops.decode_attention(*args, out, num_heads, num_kv_heads, head_dim, cache.page_size, scale, window,
                             max_ctx=reach, mods=mods, keep=keep)
    if has_prefill:
        # tcgen05 (S and O in tensor memory) for the head sizes it is written for, mma.sync otherwise
        # (combinations of kept keys and score modifiers that the tcgen05 kernel has no instance for: mma.sync)
        tc = (head_dim in (64, 128) and cache.page_size >= 8 and q_stride % 8 == 0 and _prefill_backend == "tcgen05"
              and (mods is None or mods.tcgen05_takes(keep)))
        fn = ops.prefill_attention_tc if tc else ops.prefill_attention
        # the rows that are portions, and their tokens: the launch is laid out for those, not for every decoding row
        work = None if kinds is None else (kinds[1], kinds[2])
        fn(*args, ctx.num_tokens, out, num_heads, num_kv_heads, head_dim, cache.page_size, scale, window,
           min_q_len=min_q_len, work=work, mods=mods, keep=keep)
    return out
