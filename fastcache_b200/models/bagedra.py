"""Bagedra: decoder of latent-attention, gated-linear-attention and gated-delta-rule layers in any order.

Every sublayer reads the residual stream itself and its output is normed before it is added, x <- x + norm(f(x)).
The stream is kept in fp32; the copy of it in the model's dtype that the next sublayer's projections read comes
from the kernel that adds the previous sublayer's output.  Sizes, layer order and constants come from the config's
`layers` list (one dict per layer: `type`, `mixer`, `mlp`), tensor names from `l<i>.mix.*` / `l<i>.mlp.*`.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.layer_cache import LayerCache
from ..layers.embed_head import ParallelLMHead, VocabParallelEmbedding
from ..layers.latent_attention import LatentAttention
from ..layers.linear import PackedLinear, pad8
from ..layers.recurrent import GatedDeltaRule, GatedLinearAttention, fp32_vector
from ..parallel import tp as tpmod


class BagedraMLP(nn.Module):
    """GEGLU feed-forward (tanh form of gelu) whose three projections have biases."""

    def __init__(self, width: int, ff: int):
        super().__init__()
        self.ff = ff
        self.gate_up = PackedLinear(width, {"gate": ff, "up": ff}, bias=True)
        self.down = PackedLinear(ff, {"down": width}, bias=True)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        p = self.gate_up
        return ops.hybrid.linear_gelu_mul(h, p.weight, p.bias, p.offset["up"], self.ff)


class BagedraLayer(nn.Module):
    def __init__(self, mix: nn.Module, mlp: Optional[BagedraMLP], width: int, eps: float):
        super().__init__()
        self.eps = eps
        self.mix = mix
        self.norm1 = fp32_vector(width)
        self.mlp = mlp
        self.norm2 = fp32_vector(width) if mlp is not None else None

    def forward(self, positions: torch.Tensor, h: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
        """Adds both sublayers to `x` in place; returns its copy in the model's dtype."""
        a = self.mix(positions, h)
        h = ops.hybrid.linear_post_norm_add(a, self.mix.o_proj.weight, None, x, self.norm1, self.eps)
        if self.mlp is not None:
            down = self.mlp.down
            h = ops.hybrid.linear_post_norm_add(self.mlp(h), down.weight, down.bias, x, self.norm2, self.eps)
        return h


def _mixer(kind: str, m: dict, width: int, eps: float, shapes: dict, mixers: List[nn.Module]) -> nn.Module:
    if kind == "latent_attention":
        src = m.get("kv_from")
        owner = None if src is None else mixers[int(src)]
        if owner is not None and (not isinstance(owner, LatentAttention) or owner.owner[0] is not None):
            raise ValueError(f"kv_from {src} is not a latent-attention layer with cache rows of its own")
        return LatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"],
                               m["rot"]["base"], m["rot"]["dims"], eps, owner)
    if kind == "gla":
        return GatedLinearAttention(width, m["heads"], m["dim"], m["vdim"], shapes["rank"], m["tau"], eps)
    if kind == "delta":
        return GatedDeltaRule(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], eps)
    raise ValueError(f"unknown mixer type {kind!r}")


class BagedraForCausalLM(nn.Module):
    supports_compression = False            # no layer keeps per-head K/V rows
    DEFAULT_DECAY_RANK = 16                 # of `a1` where neither a checkpoint nor the config gives it

    def __init__(self, cfg):
        super().__init__()
        if tpmod.get_tp_size() > 1:
            raise ValueError("Bagedra runs on one GPU: its layers are not sharded")
        self.config = cfg
        self.width, self.vocab = cfg.width, cfg.vocab
        self.eps = float(cfg.norm["eps"])
        self.embed_scale = float(cfg.embedding["scale"])
        wide = pad8(self.width)
        self.embed = VocabParallelEmbedding(self.vocab, wide)
        self.embed.weight.weight_loader = self._load_table
        mixers: List[nn.Module] = []
        layers = []
        shapes = getattr(cfg, "checkpoint_shapes", None) or {}
        for i, entry in enumerate(cfg.layers):
            a1 = shapes.get(f"l{i}.mix.a1")
            rank = a1[0] if a1 else entry["mixer"].get("rank", self.DEFAULT_DECAY_RANK)
            mix = _mixer(entry["type"], entry["mixer"], self.width, self.eps, {"rank": rank}, mixers)
            mixers.append(mix)
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            layers.append(BagedraLayer(mix, None if mlp is None else BagedraMLP(self.width, mlp["ff"]), self.width,
                                       self.eps))
        self.layers = nn.ModuleList(layers)
        self.norm = fp32_vector(self.width)
        self.lm_head = ParallelLMHead(pad8(self.vocab), wide)
        self.lm_head.num_embeddings = self.vocab
        self.lm_head.weight.weight_loader = self._load_table
        self.checkpoint_map = self._checkpoint_map()

    # ------------------------------------------------------------------ forward
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        x, h = ops.hybrid.embed_scaled(input_ids, self.embed.weight, self.width, self.embed_scale)
        for layer in self.layers:
            h = layer(positions, h, x)
        return ops.hybrid.rms_norm_wide(x, self.norm, self.eps, h.shape[1], h.dtype)

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.lm_head(hidden)

    # ------------------------------------------------------------------ cache
    def cache_layout(self) -> List[LayerCache]:
        out = []
        for layer in self.layers:
            mix = layer.mix
            if isinstance(mix, LatentAttention):
                if mix.row_width:
                    out.append(LayerCache(mix, row_width=mix.row_width))
            else:
                out.append(LayerCache(mix, state=mix.state_shapes()))
        return out

    # ------------------------------------------------------------------ weights
    def _load_table(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        if loaded.shape != (self.vocab, self.width):
            raise ValueError(f"shape mismatch: {tuple(loaded.shape)} for a table of {(self.vocab, self.width)}")
        param.data[: self.vocab, : self.width].copy_(loaded)

    def _tensors(self):
        """(checkpoint name, parameter name, shard id, shape) of every tensor of the checkpoint."""
        W = self.width
        yield "embed", "embed.weight", None, (self.vocab, W)
        for i, layer in enumerate(self.layers):
            src, dst, mix = f"l{i}.", f"layers.{i}.", layer.mix

            def packed(owner, attr, prefix):
                for n, size in owner.sizes.items():
                    yield src + prefix + n, f"{dst}{attr}.weight", n, (size, owner.input_size)
                    if owner.bias is not None:
                        yield f"{src}{prefix}{n}.b", f"{dst}{attr}.bias", n, (size,)

            def plain(name, attr):
                return src + name, dst + attr, None, tuple(self.get_parameter(dst + attr).shape)

            yield plain("norm1", "norm1")
            yield from packed(mix.in_proj, "mix.in_proj", "mix.")
            yield from packed(mix.o_proj, "mix.o_proj", "mix.")
            if isinstance(mix, LatentAttention):
                yield from packed(mix.kv_proj, "mix.kv_proj", "mix.")
                if mix.kv_norm is not None:
                    yield plain("mix.dkv.norm", "mix.kv_norm")
            else:
                yield plain("mix.norm", "mix.norm")
            if isinstance(mix, GatedLinearAttention):
                yield from packed(mix.a2, "mix.a2", "mix.")
                yield plain("mix.a2.b", "mix.z_bias")
            if isinstance(mix, GatedDeltaRule):
                for n in ("q", "k", "v"):
                    yield f"{src}mix.{n}.conv", dst + "mix.conv", n, (mix.in_proj.sizes[n], mix.taps)
                yield plain("mix.A_log", "mix.a_log")
                yield plain("mix.dt_bias", "mix.dt_bias")
            if layer.mlp is not None:
                yield plain("norm2", "norm2")
                yield from packed(layer.mlp.gate_up, "mlp.gate_up", "mlp.")
                yield from packed(layer.mlp.down, "mlp.down", "mlp.")
        yield "final.norm", "norm", None, (W,)
        yield "head", "lm_head.weight", None, (self.vocab, W)

    def _checkpoint_map(self) -> Dict[str, Tuple[str, Optional[str]]]:
        return {name: (param, shard) for name, param, shard, _ in self._tensors()}

    def hf_weight_shapes(self, cfg) -> Dict[str, Tuple[int, ...]]:
        """Tensor names and shapes of the checkpoint of this model."""
        return {name: shape for name, _, _, shape in self._tensors()}

    def finalize_weights(self) -> None:
        for layer in self.layers:
            if isinstance(layer.mix, LatentAttention):
                layer.mix.finalize()
