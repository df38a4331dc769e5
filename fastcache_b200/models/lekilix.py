"""Lekilix: decoder of windowed-attention and matrix-memory layers in any order, some of which run several times in a row.

A layer has one norm (weight stored around zero) whose output feeds the mixer and the feed-forward side by side; their
sum is added to the residual stream, which is kept in fp32.  The projections of both sublayers are one packed product on
the way in and, where the feed-forward is dense, one on the way out; the kernel that adds to the stream also norms it for the next layer.
A loop of layers starts every pass with x <- W [x; x0], x0 being the embedding output; passes share the weights
and have their own cache.  Sizes, order and constants come from the config, tensor names from `l<i>.mix.*` / `l<i>.mlp.*`.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.layer_cache import LayerCache, PassCache
from ..layers.embed_head import ParallelLMHead, VocabParallelEmbedding
from ..layers.linear import JoinedLinear, PackedLinear, pad8
from ..layers.moe import Experts, TableRouter
from ..layers.recurrent import MatrixMemory, fp32_vector
from ..layers.windowed_attention import WindowedAttention
from ..ops.hybrid import GluSpec
from ..parallel import tp as tpmod
from ..utils.context import get_context


def one_plus(param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
    """Norm weights are stored around zero and used as 1 + w."""
    if param.data.shape != loaded.shape:
        raise ValueError(f"shape mismatch {tuple(param.data.shape)} vs {tuple(loaded.shape)}")
    param.data.copy_(loaded.float() + 1.0)


def _norm(width: int) -> nn.Parameter:
    w = fp32_vector(width)
    w.data.fill_(1.0)
    w.weight_loader = one_plus
    return w


def _mixer(kind: str, m: dict, eps: float) -> nn.Module:
    if kind == "attention":
        if m.get("vdim", m["dim"]) != m["dim"]:
            raise ValueError(f"keys of {m['dim']} cannot be values of {m['vdim']}")
        mask = m.get("mask") or {}
        return WindowedAttention(m["heads"], m["kv_heads"], m["dim"], m["scale"], mask.get("size") or 0, m["rot"]["base"],
                                 m["rot"]["dims"], eps)
    if kind == "mlstm":
        return MatrixMemory(m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps)
    raise ValueError(f"unknown mixer type {kind!r}")


class LekilixLayer(nn.Module):
    """Mixer and feed-forward on the same normed input; `mlp`: the config's entry, or None."""

    def __init__(self, kind: str, mixer: dict, mlp: Optional[dict], width: int, vocab: int, eps: float):
        super().__init__()
        self.eps = eps
        self.norm1 = _norm(width)
        self.mix = _mixer(kind, mixer, eps)
        self.ff = self.experts = None
        sizes, outs = dict(self.mix.sizes), {"o": self.mix.out_width}
        if mlp is not None and mlp["kind"] == "dense":
            self.ff = int(mlp["ff"])
            sizes.update(gate=self.ff, up=self.ff)
            outs["down"] = self.ff
        elif mlp is not None and mlp["kind"] == "moe":
            r, e = mlp["router"], mlp["expert"]
            self.router = TableRouter(vocab, r["experts"], r["top"])
            self.experts = Experts(width, r["experts"], e["ff"], GluSpec("clamped", float(e["limit"])))
        elif mlp is not None:
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        wide = self.mix.wide
        self.in_proj = PackedLinear(width, sizes, tight=wide[1:])
        self.out_proj = JoinedLinear(outs, width)
        o = self.in_proj.offset
        self.mix.bind(o)
        self.wide = (o[wide[0]], sum(sizes[n] for n in wide)) if wide else None

    def forward(self, positions: torch.Tensor, h: torch.Tensor, x: torch.Tensor, cache: PassCache, route,
                next_norm: Optional[torch.Tensor], out: Optional[torch.Tensor]) -> torch.Tensor:
        """Adds both sublayers to `x` in place; returns it normed with `next_norm` (None: as it is) in the model's dtype."""
        hy, inp, off = ops.hybrid, self.in_proj, self.in_proj.offset
        a = h.new_empty(h.shape[0], self.out_proj.input_size)
        # many rows: the dense feed-forward is a product of its own, with the gate in its epilogue
        split = self.ff is not None and h.shape[0] > hy.SMALL_ROWS
        p = hy.project(h, inp.weight, get_context(), off["gate"] if split else None, self.wide)
        self.mix(positions, p, cache, a[:, :pad8(self.mix.out_width)])
        y = None
        if self.ff is not None:
            act = a[:, self.out_proj.offset["down"]:]
            if split:
                hy.linear_glu(h, inp.weight[off["gate"]:], off["up"] - off["gate"], self.ff, GluSpec(), act)
            else:
                hy.glu(p, off["gate"], off["up"], self.ff, GluSpec(), act)
        elif self.experts is not None:
            y = self.experts(h, route)
        return hy.linear_add_norm(a, self.out_proj.weight, x, next_norm, self.eps, experts=y, out=out)


class LekilixForCausalLM(nn.Module):
    supports_compression = False            # rows leave the window by themselves, states have a fixed size

    def __init__(self, cfg):
        super().__init__()
        if tpmod.get_tp_size() > 1:
            raise ValueError("Lekilix runs on one GPU: its layers are not sharded")
        self.config = cfg
        self.width, self.vocab = cfg.width, cfg.vocab
        self.eps = float(cfg.norm["eps"])
        self.embed_scale = float(cfg.embedding["scale"])
        self.wide = pad8(self.width)
        self.embed = VocabParallelEmbedding(self.vocab, self.wide)
        self.embed.weight.weight_loader = self._load_table
        self.layers = nn.ModuleList(LekilixLayer(e["type"], e["mixer"], e.get("mlp"), self.width, self.vocab, self.eps)
                                    for e in cfg.layers)
        self.norm = _norm(self.width)
        self.lm_head = ParallelLMHead(pad8(self.vocab), self.wide)
        self.lm_head.num_embeddings = self.vocab
        self.lm_head.weight.weight_loader = self._load_table
        # runs: (layer, whether a pass of the loop starts with it, what this run keeps between steps)
        n, loop = len(self.layers), getattr(cfg, "loop", None)
        order = [(i, False) for i in range(n)]
        self.loop_in = None
        if loop:
            a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
            if not (0 <= a < b <= n and times > 0):
                raise ValueError(f"loop over layers {a} .. {b - 1}, {times} times, of {n} layers")
            self.loop_in = JoinedLinear({"x": self.width, "x0": self.width}, self.width)
            order = order[:a] + [(i, i == a) for _ in range(times) for i in range(a, b)] + order[b:]
        self._layout = [self.layers[i].mix.cache() for i, _ in order]
        self.runs = [(i, enter, c.module) for (i, enter), c in zip(order, self._layout)]
        self.checkpoint_map = {name: (param, shard) for name, param, shard, _ in self._tensors()}

    # ------------------------------------------------------------------ forward
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        hy = ops.hybrid
        x, h = hy.embed_scaled(input_ids, self.embed.weight, self.width, self.embed_scale)
        pair = left = None
        if self.loop_in is not None:                        # [x | x0], the input of the product before every pass
            pair = h.new_empty(h.shape[0], 2 * self.wide)
            left = pair[:, :self.wide]
            pair[:, self.wide:] = h
            if self.runs[0][1]:
                left.copy_(h)
        if not self.runs[0][1]:
            h = hy.rms_norm_wide(x, self.layers[self.runs[0][0]].norm1, self.eps, self.wide, h.dtype)
        routes = {i: layer.router(input_ids) for i, layer in enumerate(self.layers) if layer.experts is not None}
        for k, (i, enter, cache) in enumerate(self.runs):
            layer = self.layers[i]
            if enter:
                h = hy.linear_add_norm(pair, self.loop_in.weight, x, layer.norm1, self.eps, add=False)
            nxt = self.runs[k + 1] if k + 1 < len(self.runs) else None
            if nxt is None:
                norm, out = self.norm, None
            else:
                norm, out = (None, left) if nxt[1] else (self.layers[nxt[0]].norm1, None)
            h = layer(positions, h, x, cache, routes.get(i), norm, out)
        return h

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.lm_head(hidden)

    # ------------------------------------------------------------------ cache
    def cache_layout(self) -> List[LayerCache]:
        return self._layout

    # ------------------------------------------------------------------ weights
    def _load_table(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        if loaded.shape != (self.vocab, self.width):
            raise ValueError(f"shape mismatch: {tuple(loaded.shape)} for a table of {(self.vocab, self.width)}")
        param.data[: self.vocab, : self.width].copy_(loaded)

    def _tensors(self):
        """(checkpoint name, parameter name, shard id, shape) of every tensor of the checkpoint."""
        W = self.width
        yield "embed", "embed.weight", None, (self.vocab, W)
        if self.loop_in is not None:
            yield "loop.in", "loop_in.weight", None, (W, 2 * W)
        for i, layer in enumerate(self.layers):
            src, dst = f"l{i}.", f"layers.{i}."
            yield src + "norm1", dst + "norm1", None, (W,)
            for n, size in layer.in_proj.sizes.items():
                yield src + ("mlp." if n in ("gate", "up") else "mix.") + n, dst + "in_proj.weight", n, (size, W)
            for n, size in layer.out_proj.sizes.items():
                yield src + ("mlp." if n == "down" else "mix.") + n, dst + "out_proj.weight", n, (W, size)
            for n, attr in layer.mix.vectors.items():
                yield f"{src}mix.{n}", f"{dst}mix.{attr}", None, tuple(getattr(layer.mix, attr).shape)
            if layer.experts is not None:
                F = layer.experts.ff
                for e in range(layer.experts.count):
                    for n in ("gate", "up", "down"):
                        yield (f"{src}mlp.e{e}.{n}", f"{dst}experts.{'down' if n == 'down' else 'gate_up'}", (e, n),
                               (W, F) if n == "down" else (F, W))
                yield f"{src}mlp.table", f"{dst}router.table", None, tuple(layer.router.table.shape)
        yield "final.norm", "norm", None, (W,)
        yield "head", "lm_head.weight", None, (self.vocab, W)

    def hf_weight_shapes(self, cfg) -> Dict[str, Tuple[int, ...]]:
        """Names and shapes of the checkpoint's floating-point tensors (tables keep their initial spread)."""
        return {name: shape for name, _, _, shape in self._tensors() if not name.endswith(".table")}
