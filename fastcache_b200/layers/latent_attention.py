"""Latent attention: the cache keeps one normed latent and one rotated key part per token, shared by all heads.

Keys and values are linear in the latent.  Prefill expands the cache rows of a request to per-head keys and values;
decode moves the expansion to the other side instead (queries into the latent space, outputs out of it) and reads
the cache rows as they are.  A layer may own its rows or read those of an earlier layer.

Options: queries that come from a normed latent of their own, a sliding window, a sink per head, rotation of neighbours
instead of halves, an output gate with one number per head instead of one per column.
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn

from .. import ops
from ..engine.layer_cache import LayerCache
from ..ops.hybrid import LatentDims
from ..utils.context import get_context
from .linear import PackedLinear, pad8
from .recurrent import fp32_vector


class LatentAttention(nn.Module):
    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, scale: float,
                 rope_base: float, rope_dims: int, eps: float, owner: Optional["LatentAttention"] = None, q_rank: int = 0,
                 window: int = 0, half: bool = True, head_gate: bool = False, sink: bool = False):
        super().__init__()
        if owner is not None and (owner.dims.rank, owner.dims.rot) != (kv_rank, rot_dim):
            raise ValueError("a layer that shares cache rows needs the same latent and rotated sizes as their owner")
        self.eps = eps
        self.owner = (owner,)                     # in a tuple: not a submodule of this layer
        if rope_dims % 2 or rope_dims > rot_dim:
            raise ValueError(f"{rope_dims} rotated dimensions of a rotated part of {rot_dim}")
        q = heads * (dim + rot_dim)
        sizes = {"dq": q_rank} if q_rank else {"q": q}
        self.q_norm = fp32_vector(q_rank) if q_rank else None
        if q_rank:
            self.q_norm.data.fill_(1.0)
        self.q_proj = PackedLinear(q_rank, {"uq": q}) if q_rank else None
        self.sink = fp32_vector(heads) if sink else None
        if owner is None:
            sizes["dkv"] = kv_rank + rot_dim
            self.kv_norm = fp32_vector(kv_rank)
            self.kv_norm.data.fill_(1.0)
        else:
            self.kv_norm = None
        sizes["g"] = heads if head_gate else heads * vdim
        self.in_proj = PackedLinear(width, sizes)
        self.kv_proj = PackedLinear(kv_rank, {"uk": heads * dim, "uv": heads * vdim})
        self.o_proj = PackedLinear(heads * vdim, {"o": width})
        o = self.in_proj.offset
        self.dims = LatentDims(heads, dim, rot_dim, vdim, kv_rank, float(scale), rope_dims,
                               o.get("q", 0), o["g"], o.get("dkv"), o.get("dq"), q_rank, int(window), half, head_gate)
        freq = ops.hybrid.rope_turns(rope_base, rope_dims)
        self.register_buffer("freq", freq.to(self.o_proj.weight.device), persistent=False)
        self.row_width = pad8(kv_rank + rot_dim) if owner is None else 0
        self.rows: Optional[torch.Tensor] = None            # [blocks, block, row_width], bound by the runner
        self.w_ukt: Optional[torch.Tensor] = None
        self.w_uv: Optional[torch.Tensor] = None

    def cache(self) -> Optional[LayerCache]:
        return LayerCache(self, row_width=self.row_width) if self.row_width else None

    def finalize(self) -> None:
        """Per-head forms of the expansion weights for the absorbed computation."""
        d, w, off = self.dims, self.kv_proj.weight.data, self.kv_proj.offset
        uk = w[off["uk"]:off["uk"] + d.heads * d.dim, : d.rank].reshape(d.heads, d.dim, d.rank)
        uv = w[off["uv"]:off["uv"] + d.heads * d.vdim, : d.rank].reshape(d.heads, d.vdim, d.rank)
        self.w_ukt = uk.transpose(1, 2).contiguous()
        self.w_uv = uv.contiguous()

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        owner = self.owner[0]
        rows = self.rows if owner is None else owner.rows
        if rows is None:
            raise RuntimeError("latent attention used before its cache rows were bound")
        return ops.hybrid.latent_attention(h, self.in_proj.weight, self.dims, self.freq, self.kv_norm, self.eps,
                                           self.kv_proj, self.w_ukt, self.w_uv, rows, positions, get_context(), self.q_norm,
                                           None if self.q_proj is None else self.q_proj.weight, self.sink)
