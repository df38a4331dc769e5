"""Step metadata shared by the layers of one forward pass.

Parity: nanovllm/utils/context.py:6-28 (a process-global record of
prefill/decode metadata).  Fields here describe the paged layout directly:
`kv_lens` is the number of rows each request has in the pool after this step's
store, for prefill and decode alike.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Sequence, Tuple

import numpy as np
import torch


@dataclass
class Context:
    is_prefill: bool = False
    cu_seqlens_q: Optional[torch.Tensor] = None
    cu_seqlens_k: Optional[torch.Tensor] = None
    max_seqlen_q: int = 0
    max_seqlen_k: int = 0
    slot_mapping: Optional[torch.Tensor] = None
    context_lens: Optional[torch.Tensor] = None     # kv rows per request (decode and prefill)
    block_tables: Optional[torch.Tensor] = None
    # rows of the flattened batch whose hidden state feeds the LM head
    logits_indices: Optional[torch.Tensor] = None
    # SnapKV: when set, attention layers stash the last `window` rotated queries
    # of every request here, keyed by layer index
    window_q: Any = None
    obs_window: int = 0
    attn_workspace: Any = None
    tp: Any = None
    # models with recurrent or latent-attention layers: the state slot of every request (-1: padding row of a
    # captured batch) and, in prefill, the request and the visible rows (position + 1) of every flat row
    state_slots: Optional[torch.Tensor] = None
    row_seq: Optional[torch.Tensor] = None
    row_ctx: Optional[torch.Tensor] = None
    # latent attention in prefill: first row of every request in the batch's gathered cache rows, their total
    cu_seqlens_kv: Optional[torch.Tensor] = None
    total_kv: int = 0
    # the same on the host: rows of every request in this step and after it
    q_lens: Optional[Sequence[int]] = None
    kv_lens: Optional[Sequence[int]] = None
    _spans: Dict[int, Tuple[Any, int, int]] = field(default_factory=dict)

    def kv_span(self, window: int) -> Tuple[Optional[torch.Tensor], int, int]:
        """The last cache rows of every request that its rows of this step see through a window (0: all): (boundaries, most
        rows of a request, total)."""
        if window <= 0 or self.kv_lens is None:
            return self.cu_seqlens_kv, int(self.max_seqlen_k), int(self.total_kv)
        if window not in self._spans:
            n = np.minimum(np.asarray(self.kv_lens), np.asarray(self.q_lens) + window - 1)
            cu = torch.from_numpy(np.concatenate([[0], np.cumsum(n)]).astype(np.int32))
            if self.cu_seqlens_kv.is_cuda:
                cu = cu.pin_memory().to(self.cu_seqlens_kv.device, non_blocking=True)
            self._spans[window] = cu, int(n.max()), int(n.sum())
        return self._spans[window]


_CONTEXT = Context()


def get_context() -> Context:
    return _CONTEXT


def set_context(is_prefill: bool, cu_seqlens_q=None, cu_seqlens_k=None, max_seqlen_q=0, max_seqlen_k=0,
                slot_mapping=None, context_lens=None, block_tables=None, logits_indices=None,
                window_q=None, obs_window=0, attn_workspace=None, tp=None, **layer_fields) -> Context:
    global _CONTEXT
    _CONTEXT = Context(is_prefill, cu_seqlens_q, cu_seqlens_k, max_seqlen_q, max_seqlen_k,
                       slot_mapping, context_lens, block_tables, logits_indices, window_q,
                       obs_window, attn_workspace, tp, **layer_fields)
    return _CONTEXT


def reset_context() -> None:
    global _CONTEXT
    _CONTEXT = Context()
