"""Hyper-connections: several residual streams in place of one (Zhu et al., "Hyper-Connections")."""
from __future__ import annotations

import torch
from torch import nn


class HyperConnection(nn.Module):
    """How one sublayer reads and writes the streams: it reads sum_s in[s] x_s and afterwards x_t = sum_s mix[s, t] x_s +
    out[t] y.  One fp32 vector holds in, out and mix (from * streams + to), the form the kernels take."""

    def __init__(self, streams: int):
        super().__init__()
        self.streams = streams
        S = streams
        self.parts = {"in": (0, (S,)), "out": (S, (S,)), "mix": (2 * S, (S, S))}      # first element, shape
        start = torch.cat([torch.full((S,), 1.0 / S), torch.ones(S), torch.eye(S).flatten()])
        self.weight = nn.Parameter(start.to(torch.float32), requires_grad=False)
        self.weight.weight_loader = self._load

    def _load(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        at, shape = self.parts[shard_id]
        if loaded.shape != shape:
            raise ValueError(f"shape mismatch: {tuple(loaded.shape)} for `{shard_id}` of {self.streams} streams")
        param.data[at:at + loaded.numel()].copy_(loaded.flatten())
