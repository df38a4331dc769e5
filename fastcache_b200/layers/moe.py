"""Mixture of experts: gated feed-forward experts, one that every token uses, and routers: by a table of the token ids, by
sigmoid scores within groups, by logits."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..ops.hybrid import GluSpec
from ..utils.context import get_context
from .linear import PackedLinear, pad8
from .recurrent import fp32_vector


class TableRouter(nn.Module):
    """Every token id has its experts in a table [vocab, top]; they count equally."""

    def __init__(self, vocab: int, experts: int, top: int):
        super().__init__()
        if not 0 < top <= experts:
            raise ValueError(f"{top} experts per token of {experts}")
        self.experts = experts
        spread = (torch.arange(vocab)[:, None] * top + torch.arange(top)) % experts
        self.table = nn.Parameter(spread.to(torch.int32), requires_grad=False)
        self.table.weight_loader = self._load

    def _load(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        if loaded.shape != param.data.shape or loaded.is_floating_point():
            raise ValueError(f"an integer table of {tuple(param.data.shape)} expected, got {loaded.dtype} {tuple(loaded.shape)}")
        if loaded.min() < 0 or loaded.max() >= self.experts:
            raise ValueError(f"the table names experts outside 0 .. {self.experts - 1}")
        param.data.copy_(loaded)

    def forward(self, input_ids: torch.Tensor):
        """The step's routing; depends on the ids alone, so passes that run a layer again share it."""
        return ops.hybrid.route_by_table(input_ids, self.table, self.experts, get_context())


class ScoreRouter(nn.Module):
    """Experts by sigmoid scores of a linear map.  A correction per expert takes part in the choice but not in the weights;
    experts stand in equal groups of neighbours, of which the best `keep` (by their two largest choice scores) take part."""

    def __init__(self, width: int, experts: int, top: int, groups: int = 1, keep: int = 1):
        super().__init__()
        if experts % groups or not 0 < keep <= groups or not 0 < top <= keep * (experts // groups):
            raise ValueError(f"{top} experts per token from {keep} of {groups} groups of {experts} experts")
        self.experts, self.top, self.groups, self.keep = experts, top, groups, keep
        self.proj = PackedLinear(width, {"router": experts})
        self.correction = nn.Parameter(torch.zeros(experts, dtype=torch.float32), requires_grad=False)

    def forward(self, h: torch.Tensor):
        """(the step's routing, weights)"""
        return ops.hybrid.route_by_score(h, self.proj.weight, self.correction, self.top, self.groups, self.keep, get_context())


class LogitRouter(nn.Module):
    """The `top` experts with the largest logits of a linear map with bias; their weights are the softmax of these logits.
    `shared`: one more row of the map gives a shared expert's factor, through a sigmoid."""

    def __init__(self, width: int, experts: int, top: int, shared: bool = False):
        super().__init__()
        if not 0 < top <= experts:
            raise ValueError(f"{top} experts per token of {experts}")
        self.experts, self.top, self.shared = experts, top, shared
        self.proj = PackedLinear(width, dict({"router": experts}, **({"sg": 1} if shared else {})), tight=("sg",))
        self.bias = fp32_vector(experts)

    def forward(self, h: torch.Tensor):
        """(the step's routing, weights, factor of the shared expert or None)"""
        return ops.hybrid.route_by_logit(h, self.proj.weight, self.bias, self.top, self.shared, get_context())


class GatedFeedForward(nn.Module):
    """Gated feed-forward up to its down projection, without biases (a shared expert)."""

    def __init__(self, width: int, ff: int, spec: GluSpec):
        super().__init__()
        self.ff, self.spec = int(ff), spec
        self.gate_up = PackedLinear(width, {"gate": self.ff, "up": self.ff})
        self.down = PackedLinear(self.ff, {"down": width})

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        a = h.new_empty(h.shape[0], pad8(self.ff))
        ops.hybrid.linear_glu(h, self.gate_up.weight, self.gate_up.offset["up"], self.ff, self.spec, a)
        return a


class Experts(nn.Module):
    """Gated feed-forward experts without biases, stacked: [E, gate rows | up rows, width] and [E, width, ff]."""

    def __init__(self, width: int, experts: int, ff: int, spec: GluSpec):
        super().__init__()
        self.width, self.count, self.ff, self.spec = width, experts, ff, spec
        fp = pad8(ff)
        self.gate_up = nn.Parameter(torch.zeros(experts, 2 * fp, pad8(width)), requires_grad=False)
        self.gate_up.weight_loader = self._load
        self.down = nn.Parameter(torch.zeros(experts, pad8(width), fp), requires_grad=False)
        self.down.weight_loader = self._load

    def _load(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        e, name = shard_id
        at = pad8(self.ff) if name == "up" else 0
        want = (self.width, self.ff) if name == "down" else (self.ff, self.width)
        if loaded.shape != want:
            raise ValueError(f"shape mismatch: {tuple(loaded.shape)} for {name} of {want}")
        param.data[e, at:at + want[0], :want[1]].copy_(loaded)

    def forward(self, h: torch.Tensor, route, weights=None):
        return ops.hybrid.experts(h, route, weights, self.gate_up, self.down, self.ff, self.spec)
