"""Rotary position encoding, rotate-half pairing (inference_engine/model.py:56-69).

Parameters: the head size, how many leading dimensions rotate (``rotary_dim``; the reference
rotates all of them), the base ``theta`` and the table length.  ``inv_freq[j] = theta^(-2j/rotary_dim)``
and the angles p * inv_freq[j] are float32; cos/sin tables are float32 too (the reference rounds
them to the model dtype, inference_engine/model.py:61).  The rotation is fused with the write of
keys and values into their cache slots, which the reference does right after it
(inference_engine/model.py:130-134).

``NoPosition`` is the same interface for a mixer without position encoding: it only stores.
"""
from __future__ import annotations

import math
import os

import torch

from ..kernels import ops
from .base import Part, register_part

_table_cache: dict = {}
ROTATE_IN_ATTENTION = os.environ.get("MIE_B200_ROPE_IN_ATTENTION", "1") != "0"


class Rope(Part):
    def __init__(self, head_dim: int, rotary_dim: int, theta: float, max_position: int):
        if rotary_dim % 2 or rotary_dim > head_dim or rotary_dim < 0:
            raise ValueError(f"rotary_dim {rotary_dim} must be even and at most head_dim {head_dim}")
        self.head_dim = head_dim
        self.rotary_dim = rotary_dim
        self.theta = float(theta)
        self.max_position = max_position

    def kernel_sources(self):
        return {"rope_cache"}

    def inv_freq(self) -> torch.Tensor:
        j = torch.arange(0, self.rotary_dim, 2, dtype=torch.int64).float()
        return 1.0 / (self.theta ** (j / self.rotary_dim))

    def bind(self, tensors, rt):
        self.rt = rt
        key = (str(rt.device), self.rotary_dim, self.theta, self.max_position)
        if key not in _table_cache:
            if self.rotary_dim:
                _table_cache[key] = ops.rope_tables(self.inv_freq().to(rt.device), self.max_position)
            else:
                z = torch.zeros(self.max_position, 0, dtype=torch.float32, device=rt.device)
                _table_cache[key] = (z, z)
        self.cos, self.sin = _table_cache[key]

    def project_rotate_and_store(self, x, w_qkv, b_qkv, ctx, cache, num_heads, num_kv_heads):
        """The q|k|v projection followed by rotate_and_store.  Where the tensor-core product can do
        the rotation and the cache write in its epilogue (few tokens, bfloat16), that is one kernel."""
        from ..kernels import gemm_tc, linear as linear_kernels
        if (linear_kernels.uses_tcgen05(x, w_qkv) and cache.k is not None and cache.k.dtype == torch.bfloat16
                and gemm_tc.can_fuse_rope(x, w_qkv, num_heads, num_kv_heads, self.head_dim, self.rotary_dim)):
            qkv = self.rt.empty(x.shape[0], w_qkv.shape[0])
            if gemm_tc.supports(x, w_qkv, qkv):
                return gemm_tc.gemm_qkv_rope(x, w_qkv, qkv, b_qkv, ctx.positions, ctx.slots[cache.group], self.cos, self.sin,
                                             cache.k, cache.v, num_heads, num_kv_heads, self.head_dim, self.rotary_dim,
                                             cache.page_size, write_cache=cache.writes)
        qkv = self.rt.linear(x, w_qkv, b_qkv)
        self.rotate_and_store(qkv, ctx, cache, num_heads, num_kv_heads)
        return qkv

    def rotates_in_attention(self, x, w_qkv, ctx, cache) -> bool:
        """Whether the mixer should leave rotation and the cache write to its attention kernel (``tables``):
        a step of decoding rows only whose q|k|v product is the library's (above the token count that the
        tensor-core product with the rotating epilogue serves) -- one launch less a layer."""
        from ..kernels import attention as attn_kernels, linear as linear_kernels
        return (ROTATE_IN_ATTENTION and self.rotary_dim == self.head_dim and cache.k is not None and cache.writes
                and cache.k.dtype == torch.bfloat16 and not linear_kernels.uses_tcgen05(x, w_qkv)
                and attn_kernels.rotates_in_decode(x.dtype, self.head_dim, ctx))

    def tables(self):
        return self.cos, self.sin

    def rotate_and_store(self, qkv, ctx, cache, num_heads, num_kv_heads):
        ops.rope_cache_write(qkv, ctx.positions, ctx.slots[cache.group], self.cos, self.sin, cache.k, cache.v,
                             num_heads, num_kv_heads, self.head_dim, self.rotary_dim, cache.page_size,
                             write_cache=cache.writes)


class NoPosition(Rope):
    def __init__(self, head_dim: int, max_position: int):
        super().__init__(head_dim, 0, 1.0, max_position)


register_part("position", "rope", Rope)
register_part("position", "none", NoPosition)


def rotary_frequencies(dims: int, base: float, scaling: dict | None = None) -> torch.Tensor:
    """float32 frequencies f_i = base^(-2i/dims), i < dims/2, for kernels that compute angles from positions
    themselves (no table, no bound on the position).  ``scaling`` may rescale them; its ``kind`` says how:

    * "wavelength" (the default), {factor, low, high, original}: by wavelength l = 2 pi / f, waves shorter than original/high
      keep their frequency, waves longer than original/low get f / factor, and between the two the frequency is the blend
      (1 - s) f / factor + s f with s = (original / l - low) / (high - low);
    * "linear", {factor}: every f_i / factor;
    * "yarn", {factor, original, fast, slow}: the pair that makes t turns over ``original`` positions has the index
      d(t) = dims ln(original / (2 pi t)) / (2 ln base); pairs up to floor(d(fast)) keep their frequency, pairs from ceil(d(slow))
      on get f / factor, and between the two the share of f / factor grows linearly with the index.  (cos and sin of such a
      rotation are also scaled: ``rotary_gain``.)"""
    kind = (scaling or {}).get("kind", "wavelength")
    if kind not in ("wavelength", "linear", "yarn"):
        raise ValueError(f"rotary scaling {kind!r}; wavelength, linear or yarn")
    if scaling and kind == "yarn":
        factor, orig, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))
        index = lambda turns: dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))
        lo, hi = max(math.floor(index(fast)), 0), min(math.ceil(index(slow)), dims - 1)
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling and kind == "linear":
            f = f / float(scaling["factor"])
        elif scaling and kind == "yarn":
            share = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / factor * share + f * (1.0 - share)
        elif scaling:
            factor, low, high, orig = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > orig / low:
                f = f / factor
            elif wave >= orig / high:
                s = (orig / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float32)


def rotary_gain(scaling: dict | None) -> float:
    """What cos and sin of a rescaled rotation are multiplied by: 0.1 ln(factor) + 1 for "yarn", 1 for the others."""
    return 0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling and scaling.get("kind") == "yarn" else 1.0
