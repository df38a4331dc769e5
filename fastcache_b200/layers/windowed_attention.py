"""Grouped-query attention that sees a part of the sequence, with one norm over the whole query and the whole key projection.

`WindowedAttention`: a sliding window, a learned sink per head, keys that are also the values, interleaved rotation of a part
of each head and an output gate.  `ProjectedAttention`: values of their own projection, a sliding window or chunks, optional
biases, rotation of half against half (with YaRN scaling) and soft cap of the scores.

The layers work between a packed input projection and an output projection that their owner holds (a layer whose
sublayers run in parallel packs theirs together): `sizes` names the projections they need, `bind` tells them where these
are.
"""
from __future__ import annotations

from typing import Dict, Optional

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
        self.scale, self.window, self.rope_dims = float(scale), int(window), int(rope_dims)
        self.sizes: Dict[str, int] = {"q": heads * dim, "k": kv_heads * dim, "g": heads * dim}
        self.out_width = heads * dim
        self.q_norm = fp32_vector(heads * dim)
        self.k_norm = fp32_vector(kv_heads * dim)
        self.sink = fp32_vector(heads)
        freq = ops.hybrid.rope_turns(rope_base, rope_dims)
        self.register_buffer("freq", freq.to(self.sink.device), persistent=False)
        self.vectors = {"q.norm": "q_norm", "k.norm": "k_norm", "sink": "sink"}       # checkpoint name -> parameter

    def bind(self, offset: Dict[str, int]) -> None:
        self.dims = WindowDims(self.heads, self.kv_heads, self.dim, self.rope_dims, self.scale, self.window, offset["q"],
                               offset["k"], offset["g"])

    def cache(self) -> LayerCache:
        return LayerCache(PassCache(), kv=(self.kv_heads, padded_dim(self.dim)))

    def forward(self, positions: torch.Tensor, p, cache: PassCache, out: torch.Tensor) -> None:
        ops.hybrid.windowed_attention(p, self.dims, self.freq, self.q_norm, self.k_norm, self.sink, self.eps, cache.k_rows,
                                      cache.v_rows, positions, get_context(), out)


class ProjectedAttention(nn.Module):
    """`window` / `chunk`: see `WindowDims` (0: the whole past).  `rope`: None (positions do not enter the scores) or `base`,
    `dims` and, for YaRN, `scaling`.  `bias`: the projections have one."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, window: int = 0,
                 chunk: int = 0, softcap: float = 0.0, rope: Optional[dict] = None, bias: bool = False):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads cannot share {kv_heads} key heads evenly")
        self.heads, self.kv_heads, self.dim, self.vdim, self.eps, self.bias = heads, kv_heads, dim, vdim, eps, bias
        self.seen = dict(scale=float(scale), window=int(window), chunk=int(chunk), softcap=float(softcap or 0.0))
        self.rope_dims = int(rope["dims"]) if rope else 0
        if self.rope_dims % 2 or self.rope_dims > dim:
            raise ValueError(f"{self.rope_dims} rotated dimensions of a head of {dim}")
        self.sizes: Dict[str, int] = {"q": heads * dim, "k": kv_heads * dim, "v": kv_heads * vdim}
        self.out_width = heads * vdim
        self.q_norm = fp32_vector(heads * dim)
        self.k_norm = fp32_vector(kv_heads * dim)
        scaling = rope.get("scaling") if rope else None
        freq = ops.hybrid.rope_turns(rope["base"], self.rope_dims, scaling) if rope else torch.empty(0, dtype=torch.float64)
        self.rope_size = ops.hybrid.rope_size(scaling)
        self.register_buffer("freq", freq.to(self.q_norm.device), persistent=False)
        self.vectors = {"q.norm": "q_norm", "k.norm": "k_norm"}

    def bind(self, offset: Dict[str, int]) -> None:
        self.dims = WindowDims(self.heads, self.kv_heads, self.dim, self.rope_dims, q=offset["q"], k=offset["k"],
                               v=offset["v"], vdim=self.vdim, half=True, rot_size=self.rope_size, **self.seen)

    def cache(self) -> LayerCache:
        return LayerCache(PassCache(), kv=(self.kv_heads, padded_dim(max(self.dim, self.vdim))))

    def forward(self, positions: torch.Tensor, h: torch.Tensor, proj, cache: PassCache) -> torch.Tensor:
        """`proj`: the packed projection (q, k, v) of h."""
        ctx = get_context()
        out = h.new_empty(h.shape[0], pad8(self.out_width))
        ops.hybrid.windowed_attention(ops.hybrid.project(h, proj.weight, ctx), self.dims, self.freq, self.q_norm, self.k_norm,
                                      None, self.eps, cache.k_rows, cache.v_rows, positions, ctx, out, proj.bias)
        return out
