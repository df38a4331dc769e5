"""Darusun: decoder of attention layers with mixed heads and of latent-attention layers in any order.

Every sublayer reads the residual stream itself; its output is normed, multiplied and added, x <- x + mult * norm(f(x)).  The
stream is kept in fp32; the copy of it in the model's dtype that the next sublayer reads comes from the kernel that adds the
previous sublayer's output.  A norm has one number for all columns; with the multiplier it becomes that kernel's weight vector.
Attention layers may read an earlier layer's keys and values.  Feed-forwards are dense (xIELU) or experts with a shared one.
Sizes, order and constants come from the config, tensor names from `l<i>.mix.*` / `l<i>.mlp.*`.
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch
from torch import nn
from torch.nn import functional as F

from .. import ops
from ..engine.layer_cache import LayerCache
from ..layers.embed_head import ParallelLMHead, VocabParallelEmbedding
from ..layers.latent_attention import LatentAttention
from ..layers.linear import PackedLinear, pad8
from ..layers.moe import Experts, GatedFeedForward, LogitRouter
from ..layers.recurrent import fp32_vector
from ..layers.talking_attention import TalkingAttention
from ..ops.hybrid import GluSpec
from ..parallel import tp as tpmod


def scalar_norm(width: int, factor: float = 1.0) -> nn.Parameter:
    """Weight vector of a norm whose checkpoint tensor is one number, times `factor`."""
    w = fp32_vector(width)
    w.data.fill_(factor)

    def load(param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        if loaded.numel() != 1:
            raise ValueError(f"shape mismatch: {tuple(loaded.shape)} for a norm of one number")
        param.data.fill_(float(loaded) * factor)

    w.weight_loader = load
    return w


class XieluMLP(nn.Module):
    """Feed-forward without a gate; its activation's two numbers p, q are kept as softplus(p) and 1/2 + softplus(q)."""

    def __init__(self, width: int, mlp: dict):
        super().__init__()
        self.ff = int(mlp["ff"])
        self.up = PackedLinear(width, {"up": self.ff})
        self.down = PackedLinear(self.ff, {"down": width})
        self.coef = fp32_vector(2)
        self.coef.weight_loader = self._load
        self._load(self.coef, torch.zeros(2))

    def _load(self, param: nn.Parameter, loaded: torch.Tensor, shard_id=None) -> None:
        if loaded.shape != (2,):
            raise ValueError(f"shape mismatch: {tuple(loaded.shape)} for the two numbers of xIELU")
        c = F.softplus(loaded.double())
        param.data.copy_(c + torch.tensor([0.0, 0.5], dtype=torch.float64, device=c.device))

    def forward(self, h, x, norm_w, eps: float) -> torch.Tensor:
        a = ops.hybrid.linear_xielu(h, self.up.weight, self.coef, self.ff)
        return ops.hybrid.linear_post_norm_add(a, self.down.weight, None, x, norm_w, eps)


class ExpertsMLP(nn.Module):
    """Experts by logits beside a shared expert with a factor per token."""

    def __init__(self, width: int, mlp: dict):
        super().__init__()
        r = mlp["router"]
        self.router = LogitRouter(width, r["experts"], r["top"], shared=True)
        self.experts = Experts(width, r["experts"], int(mlp["expert"]["ff"]), GluSpec("silu"))
        self.shared = GatedFeedForward(width, mlp["shared"]["ff"], GluSpec("silu"))

    def forward(self, h, x, norm_w, eps: float) -> torch.Tensor:
        route, weights, factor = self.router(h)
        y = self.experts(h, route, weights)
        return ops.hybrid.linear_post_norm_add(self.shared(h), self.shared.down.weight, None, x, norm_w, eps, y, factor)


class DarusunLayer(nn.Module):
    def __init__(self, entry: dict, mix: nn.Module, width: int, mult: float, eps: float):
        super().__init__()
        self.eps, self.mix = eps, mix
        self.norm1 = scalar_norm(width, mult)
        mlp, self.mlp, self.norm2 = entry.get("mlp"), None, None
        if mlp is not None:
            kinds = {"dense": XieluMLP, "moe": ExpertsMLP}
            if mlp["kind"] not in kinds:
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            self.mlp, self.norm2 = kinds[mlp["kind"]](width, mlp), scalar_norm(width, mult)

    def forward(self, positions: torch.Tensor, h: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
        """Adds both sublayers to `x` in place; returns its copy in the model's dtype."""
        a = self.mix(positions, h)
        h = ops.hybrid.linear_post_norm_add(a, self.mix.o_proj.weight, None, x, self.norm1, self.eps)
        return h if self.mlp is None else self.mlp(h, x, self.norm2, self.eps)


def _mixer(kind: str, m: dict, width: int, eps: float, mixers: List[nn.Module]) -> nn.Module:
    if kind == "attention":
        src = m.get("kv_from")
        if src is not None and not 0 <= int(src) < len(mixers):
            raise ValueError(f"kv_from {src} of layer {len(mixers)}: not an earlier layer")
        owner = None if src is None else mixers[int(src)]
        if owner is not None and (not isinstance(owner, TalkingAttention) or owner.owner[0] is not None):
            raise ValueError(f"kv_from {src} is not an attention layer with cache rows of its own")
        return TalkingAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["rot"]["base"],
                                m["rot"]["dims"], eps, owner)
    if kind == "latent_attention":
        return LatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], m["rot"]["base"],
                               m["rot"]["dims"], eps, q_rank=m["q_rank"], window=int((m.get("mask") or {}).get("size") or 0), half=False,
                               head_gate=True, sink=True)
    raise ValueError(f"unknown mixer type {kind!r}")


class DarusunForCausalLM(nn.Module):
    supports_compression = False            # no layer keeps per-head K/V rows

    def __init__(self, cfg):
        super().__init__()
        if tpmod.get_tp_size() > 1:
            raise ValueError("Darusun runs on one GPU: its layers are not sharded")
        self.config = cfg
        self.width, self.vocab = cfg.width, cfg.vocab
        self.eps = float(cfg.norm["eps"])
        mult = float(cfg.residual_mult)
        wide = pad8(self.width)
        self.embed = VocabParallelEmbedding(self.vocab, wide)
        self.embed.weight.weight_loader = self._load_table
        mixers: List[nn.Module] = []
        for entry in cfg.layers:
            mixers.append(_mixer(entry["type"], entry["mixer"], self.width, self.eps, mixers))
        self.layers = nn.ModuleList(DarusunLayer(e, m, self.width, mult, self.eps) for e, m in zip(cfg.layers, mixers))
        self.norm = scalar_norm(self.width)
        self.lm_head = ParallelLMHead(pad8(self.vocab), wide)
        self.lm_head.num_embeddings = self.vocab
        self.lm_head.weight.weight_loader = self._load_table
        self._layout = [c for c in (m.cache() for m in mixers) if c is not None]
        self.checkpoint_map = {name: (param, shard) for name, param, shard, _ in self._tensors()}

    # ------------------------------------------------------------------ forward
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        x, h = ops.hybrid.embed_scaled(input_ids, self.embed.weight, self.width, 1.0)
        for layer in self.layers:
            h = layer(positions, h, x)
        return ops.hybrid.rms_norm_wide(x, self.norm, self.eps, h.shape[1], h.dtype)

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

        def packed(owner: PackedLinear, src: str, dst: str):
            for n, size in owner.sizes.items():
                yield src + n, dst + ".weight", n, (size, owner.input_size)

        yield "embed", "embed.weight", None, (self.vocab, W)
        for i, layer in enumerate(self.layers):
            mix, mlp, src, dst = layer.mix, layer.mlp, f"l{i}.mix.", f"layers.{i}.mix."
            yield f"l{i}.norm1", f"layers.{i}.norm1", None, ()
            yield from packed(mix.in_proj, src, dst + "in_proj")
            yield from packed(mix.o_proj, src, dst + "o_proj")
            if isinstance(mix, TalkingAttention):
                yield src + "talk", dst + "talk", None, tuple(mix.talk.shape)
            else:
                yield from packed(mix.q_proj, src, dst + "q_proj")
                yield from packed(mix.kv_proj, src, dst + "kv_proj")
                for n, attr in (("dq.norm", "q_norm"), ("dkv.norm", "kv_norm"), ("sink", "sink")):
                    yield src + n, dst + attr, None, tuple(getattr(mix, attr).shape)
            if mlp is None:
                continue
            src, dst = f"l{i}.mlp.", f"layers.{i}.mlp."
            yield f"l{i}.norm2", f"layers.{i}.norm2", None, ()
            if isinstance(mlp, XieluMLP):
                yield from packed(mlp.up, src, dst + "up")
                yield from packed(mlp.down, src, dst + "down")
                yield src + "act", dst + "coef", None, (2,)
                continue
            ff = mlp.experts.ff
            for e in range(mlp.experts.count):
                for n in ("gate", "up", "down"):
                    yield (f"{src}e{e}.{n}", f"{dst}experts.{'down' if n == 'down' else 'gate_up'}", (e, n),
                           (W, ff) if n == "down" else (ff, W))
            router = mlp.router.proj
            yield src + "router", dst + "router.proj.weight", "router", (router.sizes["router"], W)
            yield src + "shared.sg", dst + "router.proj.weight", "sg", (1, W)
            yield src + "router.b", dst + "router.bias", None, (router.sizes["router"],)
            yield from packed(mlp.shared.gate_up, src + "shared.", dst + "shared.gate_up")
            yield from packed(mlp.shared.down, src + "shared.", dst + "shared.down")
        yield "final.norm", "norm", None, ()
        yield "head", "lm_head.weight", None, (self.vocab, W)

    def hf_weight_shapes(self, cfg) -> Dict[str, Tuple[int, ...]]:
        """Names and shapes of the tensors that a random initialisation draws: norms, head mixes, sinks, activations and router
        biases keep their initial values."""
        keep = (".talk", ".sink", ".act", ".router.b")
        return {name: shape for name, _, _, shape in self._tensors()
                if "norm" not in name.rsplit(".", 1)[-1] and not name.endswith(keep)}

    def finalize_weights(self) -> None:
        for layer in self.layers:
            if isinstance(layer.mix, LatentAttention):
                layer.mix.finalize()
