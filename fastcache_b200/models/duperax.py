"""Duperax: decoder of attention layers (sliding window, or chunks with rotary positions) and real-gated linear recurrent
units in any order, some of which run several times in a row, on several residual streams.

Every sublayer (mixer, feed-forward) reads a weighted sum of the streams through a layer norm, and its output is spread over
the streams while they are mixed (hyper-connections).  The streams are kept in fp32; the kernel that mixes them also makes
the next sublayer's normed input, so a sublayer takes that input and returns its successor's.  Feed-forwards are dense or
experts chosen by score.  Sizes, order and constants come from the config, tensor names from `l<i>.mix.*` / `l<i>.mlp.*` /
`l<i>.hc1.*` / `l<i>.hc2.*`.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.layer_cache import LayerCache, PassCache
from ..layers.embed_head import ParallelLMHead, VocabParallelEmbedding
from ..layers.hyper_connection import HyperConnection
from ..layers.linear import PackedLinear, pad8
from ..layers.moe import Experts, ScoreRouter
from ..layers.recurrent import RealGatedLRU, fp32_vector
from ..layers.windowed_attention import ProjectedAttention
from ..ops.hybrid import GluSpec
from ..parallel import tp as tpmod


def _mixer(kind: str, m: dict, eps: float) -> nn.Module:
    if kind == "rglru":
        return RealGatedLRU(m["width"], m["blocks"], m["conv"])
    if kind in ("attention", "attention_2"):
        size = int((m.get("mask") or {}).get("size") or 0)
        sizes = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps
        if kind == "attention":
            return ProjectedAttention(*sizes, window=size)
        return ProjectedAttention(*sizes, chunk=size, softcap=m.get("softcap") or 0.0, rope=m["rot"], bias=True)
    raise ValueError(f"unknown mixer type {kind!r}")


class LayerNorm(nn.Module):
    """Weight and bias (each times `scale`) of a layer norm that the stream kernels apply."""

    def __init__(self, width: int, scale: float = 1.0):
        super().__init__()
        self.scale = scale
        self.weight, self.bias = fp32_vector(width), fp32_vector(width)
        self.weight.data.fill_(scale)
        for p in (self.weight, self.bias):
            p.weight_loader = self._load

    def _load(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        if param.data.shape != loaded.shape:
            raise ValueError(f"shape mismatch {tuple(param.data.shape)} vs {tuple(loaded.shape)}")
        param.data.copy_(loaded.float() * self.scale)


class Sublayer(nn.Module):
    """What mixer and feed-forward have in common: their connection to the streams, their norm, and the output projection."""

    def __init__(self, width: int, streams: int):
        super().__init__()
        self.hc = HyperConnection(streams)
        self.norm = LayerNorm(width)

    def entry(self):
        return self.hc.weight, self.norm.weight, self.norm.bias


class MixerSublayer(Sublayer):
    def __init__(self, kind: str, mixer: dict, width: int, streams: int, eps: float):
        super().__init__(width, streams)
        self.mix = _mixer(kind, mixer, eps)
        self.in_proj = PackedLinear(width, self.mix.sizes, bias=self.mix.bias)
        self.o_proj = PackedLinear(self.mix.out_width, {"o": width})
        self.mix.bind(self.in_proj.offset)

    def forward(self, positions, h, x, cache: PassCache, nxt, eps: float) -> torch.Tensor:
        a = self.mix(positions, h, self.in_proj, cache)
        return ops.hybrid.linear_mix_norm(a, self.o_proj.weight, x, self.hc.weight, nxt, eps, h.dtype)


class DenseSublayer(Sublayer):
    def __init__(self, mlp: dict, width: int, streams: int):
        super().__init__(width, streams)
        self.ff, self.spec = int(mlp["ff"]), GluSpec("clamped", float(mlp["limit"]))
        self.gate_up = PackedLinear(width, {"gate": self.ff, "up": self.ff})
        self.down = PackedLinear(self.ff, {"down": width})

    def forward(self, positions, h, x, cache, nxt, eps: float) -> torch.Tensor:
        a = h.new_empty(h.shape[0], pad8(self.ff))
        ops.hybrid.linear_glu(h, self.gate_up.weight, self.gate_up.offset["up"], self.ff, self.spec, a)
        return ops.hybrid.linear_mix_norm(a, self.down.weight, x, self.hc.weight, nxt, eps, h.dtype)


class ExpertsSublayer(Sublayer):
    def __init__(self, mlp: dict, width: int, streams: int):
        super().__init__(width, streams)
        r = mlp["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        self.router = ScoreRouter(width, r["experts"], r["top"], groups["count"], groups["keep"])
        self.experts = Experts(width, r["experts"], mlp["expert"]["ff"], GluSpec("silu"))

    def forward(self, positions, h, x, cache, nxt, eps: float) -> torch.Tensor:
        y = self.experts(h, *self.router(h))
        return ops.hybrid.linear_mix_norm(None, None, x, self.hc.weight, nxt, eps, h.dtype, experts=y)


class DuperaxLayer(nn.Module):
    def __init__(self, entry: dict, width: int, streams: int, eps: float):
        super().__init__()
        self.first = MixerSublayer(entry["type"], entry["mixer"], width, streams, eps)
        mlp, self.second = entry.get("mlp"), None
        if mlp is not None:
            kinds = {"dense": DenseSublayer, "moe": ExpertsSublayer}
            if mlp["kind"] not in kinds:
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            self.second = kinds[mlp["kind"]](mlp, width, streams)

    def sublayers(self) -> List[Sublayer]:
        return [self.first] if self.second is None else [self.first, self.second]


class DuperaxForCausalLM(nn.Module):
    supports_compression = False            # windows and chunks end by themselves, states have a fixed size

    def __init__(self, cfg):
        super().__init__()
        if tpmod.get_tp_size() > 1:
            raise ValueError("Duperax runs on one GPU: its layers are not sharded")
        self.config = cfg
        self.width, self.vocab, self.streams = cfg.width, cfg.vocab, int(cfg.streams)
        self.eps = float(cfg.norm["eps"])
        self.embed = VocabParallelEmbedding(self.vocab, pad8(self.width))
        self.embed.weight.weight_loader = self._load_table
        self.layers = nn.ModuleList(DuperaxLayer(e, self.width, self.streams, self.eps) for e in cfg.layers)
        # the logits' factor sits in the last norm
        self.norm = LayerNorm(self.width, float(getattr(cfg, "logit_scale", None) or 1.0))
        self.lm_head = ParallelLMHead(pad8(self.vocab), pad8(self.width))
        self.lm_head.num_embeddings = self.vocab
        self.lm_head.weight.weight_loader = self._load_table
        n, loop = len(self.layers), getattr(cfg, "loop", None)
        order = list(range(n))
        if loop:
            a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
            if not (0 <= a < b <= n and times > 0):
                raise ValueError(f"loop over layers {a} .. {b - 1}, {times} times, of {n} layers")
            order = order[:a] + order[a:b] * times + order[b:]
        self._layout = [self.layers[i].first.mix.cache() for i in order]
        # (sublayer, what this run of it keeps between steps)
        self.steps = [(sub, c.module) for i, c in zip(order, self._layout) for sub in self.layers[i].sublayers()]
        self.checkpoint_map = {name: (param, shard) for name, param, shard, _ in self._tensors()}

    # ------------------------------------------------------------------ forward
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        entries = [sub.entry() for sub, _ in self.steps] + [(None, self.norm.weight, self.norm.bias)]
        x, h = ops.hybrid.embed_streams(input_ids, self.embed.weight, self.width, self.streams, entries[0], self.eps)
        for k, (sub, cache) in enumerate(self.steps):
            h = sub(positions, h, x, cache, entries[k + 1], self.eps)
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

        def norm(src, dst):
            yield src, dst + ".weight", None, (W,)
            yield src + ".b", dst + ".bias", None, (W,)

        def packed(owner: PackedLinear, src, dst):
            for n, size in owner.sizes.items():
                yield src + n, dst + ".weight", n, (size, owner.input_size)
                if owner.bias is not None:
                    yield f"{src}{n}.b", dst + ".bias", n, (size,)

        yield "embed", "embed.weight", None, (self.vocab, W)
        for i, layer in enumerate(self.layers):
            for q, (sub, dst) in enumerate(zip(layer.sublayers(), (f"layers.{i}.first", f"layers.{i}.second")), 1):
                yield from norm(f"l{i}.norm{q}", dst + ".norm")
                for n, (_, shape) in sub.hc.parts.items():
                    yield f"l{i}.hc{q}.{n}", dst + ".hc.weight", n, shape
            first, second, src, dst = layer.first, layer.second, f"l{i}.mix.", f"layers.{i}.first."
            yield from packed(first.in_proj, src, dst + "in_proj")
            yield from packed(first.o_proj, src, dst + "o_proj")
            for n, attr in first.mix.vectors.items():
                yield src + n, f"{dst}mix.{attr}", None, tuple(getattr(first.mix, attr).shape)
            if isinstance(first.mix, RealGatedLRU):
                _, B, N, _ = first.mix.gates.shape
                for n in first.mix.GATES:
                    yield src + n, dst + "mix.gates", n, (B, N, N)
                    yield f"{src}{n}.b", dst + "mix.gate_bias", n, (B, N)
            src, dst = f"l{i}.mlp.", f"layers.{i}.second."
            if isinstance(second, DenseSublayer):
                yield from packed(second.gate_up, src, dst + "gate_up")
                yield from packed(second.down, src, dst + "down")
            elif isinstance(second, ExpertsSublayer):
                F = second.experts.ff
                for e in range(second.experts.count):
                    for n in ("gate", "up", "down"):
                        yield (f"{src}e{e}.{n}", f"{dst}experts.{'down' if n == 'down' else 'gate_up'}", (e, n),
                               (W, F) if n == "down" else (F, W))
                yield from packed(second.router.proj, src, dst + "router.proj")
                yield src + "correction", dst + "router.correction", None, (second.experts.count,)
        yield from norm("final.norm", "norm")
        yield "head", "lm_head.weight", None, (self.vocab, W)

    def hf_weight_shapes(self, cfg) -> Dict[str, Tuple[int, ...]]:
        """Names and shapes of the tensors that a random initialisation draws: connections, decays and corrections keep
        their initial values."""
        return {name: shape for name, _, _, shape in self._tensors()
                if not (".hc" in name or name.endswith((".lam", ".correction")))}
