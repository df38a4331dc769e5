"""Grouped-query attention over a sliding window with a learned sink per head, keys that are also the values, one norm
over the whole query and the whole key projection, interleaved rotation of a part of each head and an output gate.

The layer works between a packed input projection and an output projection that its owner holds (a layer whose
sublayers run in parallel packs theirs together): `sizes` names the projections it needs, `bind` tells it where they
are.
"""
from __future__ import annotations

from typing import Dict

import torch
from torch import nn

from .. import ops
from ..engine.layer_cache import LayerCache, PassCache
from ..ops.hybrid import WindowDims
from ..utils.context import get_context
from .linear import pad8
from .recurrent import fp32_vector


def padded_dim(dim: int) -> int:
    """Row width of the pages: the head sizes that the tensor-core attention kernels take, larger ones as they are."""
    return 64 if dim <= 64 else 128 if dim <= 128 else pad8(dim)


class WindowedAttention(nn.Module):
    wide = ()                                       # projections whose outputs are needed in fp32

    def __init__(self, heads: int, kv_heads: int, dim: int, scale: float, window: int, rope_base: float, rope_dims: int,
                 eps: float):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads cannot share {kv_heads} key heads evenly")
        if rope_dims % 2 or rope_dims > dim:
            raise ValueError(f"{rope_dims} rotated dimensions of a head of {dim}")
        self.eps = eps
        self.heads, self.kv_heads, self.dim = heads, kv_heads, dim
        self.scale, self.window, self.rope = float(scale), int(window), (float(rope_base), int(rope_dims))
        self.sizes: Dict[str, int] = {"q": heads * dim, "k": kv_heads * dim, "g": heads * dim}
        self.out_width = heads * dim
        self.q_norm = fp32_vector(heads * dim)
        self.k_norm = fp32_vector(kv_heads * dim)
        self.sink = fp32_vector(heads)
        freq = ops.hybrid.rope_turns(rope_base, rope_dims)
        self.register_buffer("freq", freq.to(self.sink.device), persistent=False)
        self.vectors = {"q.norm": "q_norm", "k.norm": "k_norm", "sink": "sink"}       # checkpoint name -> parameter

    def bind(self, offset: Dict[str, int]) -> None:
        self.dims = WindowDims(self.heads, self.kv_heads, self.dim, self.rope[1], self.rope[0], self.scale, self.window,
                               offset["q"], offset["k"], offset["g"])

    def cache(self) -> LayerCache:
        return LayerCache(PassCache(), kv=(self.kv_heads, padded_dim(self.dim)))

    def forward(self, positions: torch.Tensor, p, cache: PassCache, out: torch.Tensor) -> None:
        ops.hybrid.windowed_attention(p, self.dims, self.freq, self.q_norm, self.k_norm, self.sink, self.eps, cache.k_rows,
                                      cache.v_rows, positions, get_context(), out)
