"""Recurrent mixers with a fixed-size state per request: gated linear attention, the gated delta rule, matrix memory,
real-gated linear recurrent units.

They read the state that earlier steps left in the request's slot (`state`, and `conv_state` for the short
convolutions), advance it by the rows of the batch and leave it there; prefill portions of any length and decode
steps go through the same call.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.layer_cache import LayerCache, PassCache
from ..ops.hybrid import DeltaDims, GlaDims, LruDims, MatrixMemoryDims
from ..utils.context import get_context
from .linear import PackedLinear


def fp32_vector(*shape: int) -> nn.Parameter:
    """A small parameter that is used in 32-bit whatever the model's dtype."""
    return nn.Parameter(torch.zeros(*shape, dtype=torch.float32), requires_grad=False)


class GatedLinearAttention(nn.Module):
    """A memory M [dim, vdim] per head whose row r fades by its own factor at every token before the outer product of key
    and value is added; a token reads M with its query.  The factors come from a low-rank projection through
    sigmoid(.)^(1 / tau); the head outputs are RMS-normed and gated with silu."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, rank: int, tau: float, eps: float):
        super().__init__()
        self.eps = eps
        self.in_proj = PackedLinear(width, {"q": heads * dim, "k": heads * dim, "v": heads * vdim,
                                            "g": heads * vdim, "a1": rank})
        self.a2 = PackedLinear(rank, {"a2": heads * dim})
        self.z_bias = fp32_vector(heads * dim)
        self.norm = fp32_vector(vdim)
        self.o_proj = PackedLinear(heads * vdim, {"o": width})
        o = self.in_proj.offset
        self.dims = GlaDims(heads, dim, vdim, rank, float(tau), o["q"], o["k"], o["v"], o["g"], o["a1"])
        self.state: Optional[torch.Tensor] = None           # [slots, heads, dim, vdim], bound by the runner

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        d = self.dims
        return {"state": (d.heads, d.dim, d.vdim)}

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        return ops.hybrid.gla(h, self.in_proj.weight, self.dims, self.a2.weight, self.z_bias, self.norm, self.eps,
                              self.state, get_context())


class GatedDeltaRule(nn.Module):
    """A memory M [dim, vdim] per head that fades as a whole and is then corrected towards the token's value: of the
    difference between v and what M returns for k, the share `beta` is written under k; the query reads after the
    write.  q, k, v pass a short causal convolution and silu, q and k are unit vectors shared by groups of heads, fading
    and share are one number per head and token; the head outputs are RMS-normed and gated with silu."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, eps: float,
                 unit_eps: float = 1e-6):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} heads cannot share {kv_heads} q/k heads evenly")
        self.eps = eps
        self.taps = taps
        self.in_proj = PackedLinear(width, {"q": kv_heads * dim, "k": kv_heads * dim, "v": heads * vdim,
                                            "g": heads * vdim, "b": heads, "a": heads}, tight=("k", "v"))
        self.channels = 2 * kv_heads * dim + heads * vdim
        self.conv = fp32_vector(self.channels, taps)
        self.conv.weight_loader = self._load_conv
        self.a_log = fp32_vector(heads)
        self.dt_bias = fp32_vector(heads)
        self.norm = fp32_vector(vdim)
        self.o_proj = PackedLinear(heads * vdim, {"o": width})
        o = self.in_proj.offset
        self.dims = DeltaDims(heads, kv_heads, dim, vdim, o["g"], o["b"], o["a"], unit_eps)
        self.state: Optional[torch.Tensor] = None           # [slots, heads, dim, vdim], bound by the runner
        self.conv_state: Optional[torch.Tensor] = None      # [slots, taps - 1, channels]: the last inputs

    def _load_conv(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        off, size = self.in_proj.offset[shard_id], self.in_proj.sizes[shard_id]
        param.data[off:off + size].copy_(loaded)

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        d = self.dims
        return {"state": (d.heads, d.dim, d.vdim), "conv_state": (self.taps - 1, self.channels)}

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        return ops.hybrid.delta_rule(h, self.in_proj.weight, self.dims, self.conv, self.a_log, self.dt_bias,
                                     self.norm, self.eps, self.conv_state, self.state, get_context())


class MatrixMemory(nn.Module):
    """mLSTM (Beck et al., "xLSTM: Extended Long Short-Term Memory"): a memory M [dim, vdim] and a normaliser n [dim] per
    head, written with exponential gates that are kept in range by a running maximum of their logarithms (which starts
    at 0).  Gates pass a soft cap; the head outputs are RMS-normed, weighted and gated with sigmoid.

    Like `WindowedAttention` it works between projections that its owner holds."""

    wide = ("i", "f")

    def __init__(self, heads: int, dim: int, vdim: int, cap: float, eps: float):
        super().__init__()
        self.eps = eps
        self.heads, self.dim, self.vdim, self.cap = heads, dim, vdim, float(cap)
        self.sizes: Dict[str, int] = {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim, "i": heads,
                                      "f": heads}
        self.out_width = heads * vdim
        self.norm = fp32_vector(heads * vdim)
        self.i_bias = fp32_vector(heads)
        self.f_bias = fp32_vector(heads)
        self.vectors = {"norm": "norm", "i.b": "i_bias", "f.b": "f_bias"}

    def bind(self, offset: Dict[str, int]) -> None:
        self.dims = MatrixMemoryDims(self.heads, self.dim, self.vdim, self.cap, *(offset[n] for n in "qkvgif"))

    def cache(self) -> LayerCache:
        return LayerCache(PassCache(), state={"state": (self.heads, self.dim, self.vdim),
                                              "norm_state": (self.heads, self.dim), "max_state": (self.heads,)})

    def forward(self, positions: torch.Tensor, p, cache: PassCache, out: torch.Tensor) -> None:
        ops.hybrid.matrix_memory(p, self.dims, self.i_bias, self.f_bias, self.norm, self.eps, cache, get_context(), out)


class RealGatedLRU(nn.Module):
    """Recurrent block of Griffin (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient
    Language Models"): one number of state per channel that fades by a gated factor a and takes sqrt(1 - a^2) of the gated
    input.  The input passes a short causal convolution, its gates are block-diagonal matrices of it; a second branch
    (gelu) multiplies the output.  Works between projections that its owner holds."""

    def __init__(self, channels: int, blocks: int, taps: int, sharpness: float = 8.0):
        super().__init__()
        if channels % blocks:
            raise ValueError(f"{channels} channels cannot be cut into {blocks} equal parts")
        n = channels // blocks
        self.channels, self.blocks, self.taps, self.sharpness, self.bias = channels, blocks, taps, float(sharpness), True
        self.sizes: Dict[str, int] = {"y": channels, "x": channels}
        self.out_width = channels
        self.conv = fp32_vector(channels, taps)
        self.conv_bias = fp32_vector(channels)
        self.gates = nn.Parameter(torch.zeros(2, blocks, n, n), requires_grad=False)      # of the decay, of the input
        self.gates.weight_loader = self._load_gate
        self.gate_bias = fp32_vector(2, channels)
        self.gate_bias.weight_loader = self._load_gate
        self.lam = fp32_vector(channels)
        self.lam.data.copy_(torch.linspace(-7.0, -2.0, channels))
        self.vectors = {"conv": "conv", "conv.b": "conv_bias", "lam": "lam"}

    GATES = {"ra": 0, "ri": 1}

    def _load_gate(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        n = self.channels // self.blocks
        if loaded.shape != ((self.blocks, n, n) if param is self.gates else (self.blocks, n)):
            raise ValueError(f"shape mismatch: {tuple(loaded.shape)} for gates of {self.blocks} blocks of {n}")
        param.data[self.GATES[shard_id]].copy_(loaded.reshape(param.data.shape[1:]))

    def bind(self, offset: Dict[str, int]) -> None:
        self.dims = LruDims(self.channels, self.blocks, offset["y"], offset["x"], self.sharpness)

    def cache(self) -> LayerCache:
        return LayerCache(PassCache(), state={"state": (self.channels,), "conv_state": (self.taps - 1, self.channels)})

    def forward(self, positions: torch.Tensor, h: torch.Tensor, proj: PackedLinear, cache: PassCache) -> torch.Tensor:
        """`proj`: the packed projection (y, x) of h."""
        return ops.hybrid.real_gated_lru(h, proj.weight, proj.bias, self.dims, self.conv, self.conv_bias, self.gates,
                                         self.gate_bias, self.lam, cache, get_context())
