"""What the layers of a hybrid model keep between steps, and the pools that hold it.

A model whose layers do not all keep the same K/V rows describes its needs with `cache_layout()`, one `LayerCache`
per owner (a layer, or one pass through a layer that runs several times): `row_width` elements per token in pages (block
tables and slots as for K/V rows), or keys and values of `kv` = (heads, dim) in pages of the layout of the K/V pool, and
named fp32 tensors per request in state slots.  A layer that reads another layer's rows is bound to that layer's pages by
the model.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

import torch


class PassCache:
    """What one pass through a layer keeps; the attributes are bound here (k_rows and v_rows, or the named states)."""


@dataclass
class LayerCache:
    module: Any                                   # receives the tensors as attributes
    row_width: int = 0
    kv: Optional[Tuple[int, int]] = None
    state: Dict[str, Tuple[int, ...]] = field(default_factory=dict)


def state_bytes(layout: List[LayerCache]) -> int:
    """Bytes of recurrent state of one request."""
    return sum(4 * torch.Size(shape).numel() for c in layout for shape in c.state.values())


def row_bytes(layout: List[LayerCache], dtype: torch.dtype) -> int:
    """Bytes of paged rows of one token."""
    return sum(c.row_width + (2 * c.kv[0] * c.kv[1] if c.kv else 0) for c in layout) * torch.empty((), dtype=dtype).element_size()


def allocate_states(layout: List[LayerCache], num_slots: int, device: torch.device) -> None:
    """One fp32 tensor [slots, ...] per named state of every layer.  Never cleared when a slot changes hands: a run
    that starts at position 0 starts from a zero state whatever the slot holds."""
    for c in layout:
        for name, shape in c.state.items():
            setattr(c.module, name, torch.zeros(num_slots, *shape, dtype=torch.float32, device=device))


def allocate_rows(layout: List[LayerCache], num_blocks: int, block_size: int, dtype: torch.dtype,
                  device: torch.device) -> None:
    for c in layout:
        if c.row_width:
            c.module.rows = torch.zeros(num_blocks, block_size, c.row_width, dtype=dtype, device=device)
        if c.kv:
            heads, dim = c.kv
            for name in ("k_rows", "v_rows"):
                setattr(c.module, name, torch.zeros(num_blocks, heads, block_size, dim, dtype=dtype, device=device))


def release(layout: List[LayerCache]) -> None:
    for c in layout:
        for name in c.state:
            setattr(c.module, name, None)
        for name in ("rows",) if c.row_width else ("k_rows", "v_rows") if c.kv else ():
            setattr(c.module, name, None)
