"""Grouped-query attention whose heads mix their scores before the softmax (talking heads).

Queries and keys are rotated (half against half) and then brought to unit root mean square, head by head.  The cache keeps one
row per token, the keys of all key heads side by side and the values behind them: mixed scores are products of such a row with
a query that is as wide.  A layer may own its rows or read those of an earlier layer.
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn

from .. import ops
from ..engine.layer_cache import LayerCache
from ..ops.hybrid import TalkDims
from ..utils.context import get_context
from .linear import PackedLinear, pad8
from .recurrent import fp32_vector


class TalkingAttention(nn.Module):
    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, rope_base: float,
                 rope_dims: int, eps: float, owner: Optional["TalkingAttention"] = None):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads cannot share {kv_heads} key heads evenly")
        if rope_dims % 2 or rope_dims > dim:
            raise ValueError(f"{rope_dims} rotated dimensions of a head of {dim}")
        if owner is not None and (owner.dims.kv_heads, owner.dims.dim, owner.dims.vdim) != (kv_heads, dim, vdim):
            raise ValueError("a layer that shares cache rows needs the same key heads and head sizes as their owner")
        self.eps = eps
        self.owner = (owner,)                     # in a tuple: not a submodule of this layer
        sizes = {"q": heads * dim}
        if owner is None:
            sizes.update(k=kv_heads * dim, v=kv_heads * vdim)
        self.in_proj = PackedLinear(width, sizes)
        self.o_proj = PackedLinear(heads * vdim, {"o": width})
        self.talk = fp32_vector(heads, heads)
        self.talk.data.copy_(torch.eye(heads))
        freq = ops.hybrid.rope_turns(rope_base, rope_dims)
        self.register_buffer("freq", freq.to(self.talk.device), persistent=False)
        o, v_col = self.in_proj.offset, pad8(kv_heads * dim)
        self.dims = TalkDims(heads, kv_heads, dim, vdim, rope_dims, float(scale), o["q"], o.get("k"), o.get("v"), v_col)
        self.row_width = v_col + pad8(kv_heads * vdim) if owner is None else 0
        self.rows: Optional[torch.Tensor] = None            # [blocks, block, row_width], bound by the runner

    def cache(self) -> Optional[LayerCache]:
        return LayerCache(self, row_width=self.row_width) if self.row_width else None

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        owner = self.owner[0]
        rows = self.rows if owner is None else owner.rows
        if rows is None:
            raise RuntimeError("attention used before its cache rows were bound")
        ctx = get_context()
        out = h.new_empty(h.shape[0], self.o_proj.weight.shape[1])
        ops.hybrid.talking_attention(ops.hybrid.project(h, self.in_proj.weight, ctx), self.dims, self.freq, self.talk, self.eps,
                                     rows, positions, ctx, out)
        return out
