"""Ops of hybrid models (recurrent layers, latent and windowed attention, experts, norms on a 32-bit residual stream).

Same rule as the other ops of this package: the device of the data decides between the sm_100a kernels and the
PyTorch statements of `reference_hybrid.py`.  Inputs and outputs are in the model's dtype (bf16, or fp32 for runs
in 32-bit); the residual stream, the recurrent states and the small per-head vectors are always fp32.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import reference_hybrid as ref
from .loader import ext


LATENT_IMPL = 0         # tests: 1 the general kernels also where a tensor-core form exists, 2 absorbed also in prefill,
                        # 3 the same on mma.sync


def _n(k: int = 1) -> None:
    from . import COUNTERS
    COUNTERS["launches"] += k


@dataclass(frozen=True)
class GlaDims:
    """Gated linear attention: sizes, decay temperature, first columns of the packed projections."""
    heads: int
    dim: int
    vdim: int
    rank: int
    tau: float
    q: int
    k: int
    v: int
    g: int
    a1: int


@dataclass(frozen=True)
class DeltaDims:
    """Gated delta rule; q | k | v are the first columns of the packed projections, without gaps."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    g: int
    b: int
    a: int
    unit_eps: float = 1e-6


@dataclass(frozen=True)
class LatentDims:
    """Latent attention; `kv` is None for a layer that reads another layer's cache rows.

    `g` None: no output gate; `head_gate`: one column per head.  `dq`: first column of the latent (of `q_rank`) that the
    queries are made from; None: they are the columns from `q` on.  `half`: entry i of a rotated part turns with entry
    i + rot_dims / 2 (else entries 2i and 2i + 1).  `window`: the positions a query sees, itself included (0: all up to itself)."""
    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int
    scale: float
    rot_dims: int
    q: int
    g: Optional[int]
    kv: Optional[int]
    dq: Optional[int] = None
    q_rank: int = 0
    window: int = 0
    half: bool = True
    head_gate: bool = False

    def sizes(self) -> list:
        """The integers as the extension takes them (-1: no such projection)."""
        return [self.heads, self.dim, self.rot, self.vdim, self.rank, self.rot_dims, self.q, -1 if self.kv is None else self.kv,
                -1 if self.g is None else self.g, self.dq or 0, self.q_rank, self.window, int(self.half), int(self.head_gate)]


@dataclass(frozen=True)
class TalkDims:
    """Attention whose heads mix their scores: sizes, first columns of the packed projections (`k` and `v` None: another
    layer's cache rows), first value column of a cache row."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_dims: int
    scale: float
    q: int
    k: Optional[int]
    v: Optional[int]
    v_col: int

    def sizes(self) -> list:
        return [self.heads, self.kv_heads, self.dim, self.vdim, self.rot_dims, self.q, -1 if self.k is None else self.k,
                -1 if self.v is None else self.v, self.v_col]


@dataclass(frozen=True)
class WindowDims:
    """Attention over per-head rows: sizes, first columns of the packed projections, and what a query sees.

    `v` None: the values are the raw keys; `g` None: no output gate.  `half`: entry i of a head turns with entry
    i + rot_dims / 2 (else entries 2i and 2i + 1 turn together), cos and sin are multiplied by `rot_size`.  `window`: the
    positions a query sees, itself included; `chunk`: it sees no key before the last multiple of it; 0: all up to itself.
    `softcap` c > 0: scores become c tanh(score / c)."""
    heads: int
    kv_heads: int
    dim: int
    rot_dims: int
    scale: float
    window: int
    q: int
    k: int
    g: Optional[int] = None
    v: Optional[int] = None
    vdim: int = 0
    chunk: int = 0
    softcap: float = 0.0
    half: bool = False
    rot_size: float = 1.0

    @property
    def value_dim(self) -> int:
        return self.vdim or self.dim

    def sizes(self) -> list:
        """The integers as the extension takes them (-1: no such projection)."""
        return [self.heads, self.kv_heads, self.dim, self.value_dim, self.rot_dims, self.window, self.chunk, self.q, self.k,
                -1 if self.v is None else self.v, -1 if self.g is None else self.g, int(self.half)]


@dataclass(frozen=True)
class LruDims:
    """Real-gated linear recurrent unit: channels, equal parts that the gate matrices work on, first columns of the packed
    projections; the logarithm of the decay is -sharpness * r * softplus(lam)."""
    channels: int
    blocks: int
    y: int
    x: int
    sharpness: float = 8.0


@dataclass(frozen=True)
class MatrixMemoryDims:
    """Matrix memory (mLSTM): sizes, soft cap of the gates, first columns of the packed projections; `floor` is added to
    the normaliser."""
    heads: int
    dim: int
    vdim: int
    cap: float
    q: int
    k: int
    v: int
    g: int
    i: int
    f: int
    floor: float = 1e-6


@dataclass(frozen=True)
class GluSpec:
    """Gated activation: "silu", or "clamped" (see `reference_hybrid.glu`) with its limit."""
    act: str = "silu"
    limit: float = 0.0

    @property
    def code(self) -> int:
        return {"silu": 0, "clamped": 1}[self.act]


# ------------------------------------------------------------------ residual stream
def embed_scaled(ids, weight, width: int, scale: float):
    """(fp32 residual [T, width], its copy in the model's dtype [T, padded width]) of table rows times `scale`."""
    if weight.is_cuda:
        _n()
        return ext().embed_scaled(ids, weight, int(width), float(scale))
    return ref.embed_scaled(ids, weight, width, scale)


def linear_post_norm_add(a, weight, bias, x, norm_w, eps: float, experts=None, factor=None):
    """x += RMSNorm(factor * (a @ weight.T + bias) + the mixed outputs of `experts`) * norm_w in fp32, in place; returns x in
    the model's dtype (padded width).  `factor` [T] fp32, or None: 1."""
    if a.is_cuda:
        _n(2)
        y, row_of, mix = experts if experts is not None else (None, None, None)
        return ext().linear_post_norm_add(a, weight, bias, x, norm_w, float(eps), y, row_of, mix, factor)
    return ref.post_norm_add(ref_linear(a, weight, bias), x, norm_w, eps, experts, factor)


def linear_xielu(h, weight, coef, width: int):
    """xIELU of h @ weight.T (see `reference_hybrid.xielu`; coef [2] fp32), padded to 8 columns."""
    if h.is_cuda:
        _n(2)
        return ext().linear_xielu(h, weight, coef, int(width))
    z = ref_linear(h, weight)
    return ref._pad_to(ref.xielu(z[:, :width].float(), coef).to(h.dtype), z.shape[1])


def rms_norm_wide(x, norm_w, eps: float, width: int, dtype):
    """RMSNorm of the fp32 residual in the model's dtype, zero-padded to `width` columns."""
    if x.is_cuda:
        _n()
        return ext().rms_norm_wide(x, norm_w, float(eps), int(width), dtype == torch.float32)
    return ref.rms_norm_wide(x, norm_w, eps, width, dtype)


def linear_gelu_mul(h, weight, bias, up_off: int, width: int):
    """gelu_tanh(gate) * up of the packed projections gate | up (`up` from column `up_off`), padded to 8 columns."""
    if h.is_cuda:
        _n(2)
        return ext().linear_gelu_mul(h, weight, bias, int(up_off), int(width))
    return ref.gelu_tanh_and_mul(ref_linear(h, weight, bias), up_off, width)


def ref_linear(x, weight, bias=None):
    from . import linear
    return linear(x, weight, bias)


# ------------------------------------------------------------------ recurrent layers
def gla(h, weight, d: GlaDims, a2_weight, z_bias, norm_w, eps: float, state, ctx):
    """Gated linear attention of a batch of runs up to (not including) the output projection."""
    if h.is_cuda:
        _n(4)
        return ext().gla(h, weight, a2_weight, z_bias, norm_w, float(eps), state,
                         [d.heads, d.dim, d.vdim, d.rank, d.q, d.k, d.v, d.g, d.a1], float(d.tau), *_run_args(ctx))
    p = ref_linear(h, weight)
    z = ref_linear(p[:, d.a1:d.a1 + a2_weight.shape[1]], a2_weight)
    return ref.gla(p, z, d, z_bias, norm_w, eps, state, ctx)


def delta_rule(h, weight, d: DeltaDims, conv_w, a_log, dt_bias, norm_w, eps: float, conv_state, state, ctx):
    """Gated delta rule (with its short convolutions) of a batch of runs up to the output projection."""
    if h.is_cuda:
        _n(4)
        return ext().delta_rule(h, weight, conv_w, a_log, dt_bias, norm_w, float(eps), conv_state, state,
                                [d.heads, d.kv_heads, d.dim, d.vdim, d.g, d.b, d.a], float(d.unit_eps),
                                *_run_args(ctx), ctx.row_seq)
    return ref.delta_rule(ref_linear(h, weight), d, conv_w, a_log, dt_bias, norm_w, eps, conv_state, state, ctx)


def _run_args(ctx):
    """Batch layout for the recurrent kernels: run boundaries (None: one row per request), rows per request after
    this step, state slots, longest run."""
    return ctx.cu_seqlens_q, ctx.context_lens, ctx.state_slots, int(ctx.max_seqlen_q) if ctx.is_prefill else 1


# ------------------------------------------------------------------ latent attention
def latent_attention(h, weight, d: LatentDims, freq, kv_norm_w, eps: float, kv_proj, w_ukt, w_uv, pool, positions, ctx, q_norm_w=None,
                     q_weight=None, sink=None):
    """Projections, cache store, attention and output gate of a latent-attention layer up to the output projection.
    `freq`: rope_turns; `q_norm_w`, `q_weight`: norm and projection of the queries' latent; `sink` [H] joins the softmax without a key.

    `kv_proj` (packed uk | uv) expands cache rows to keys and values (prefill); `w_ukt` [H, rank, dim] and `w_uv`
    [H, vdim, rank] are the same weights for the absorbed form (decode), which never expands a row."""
    if h.is_cuda:
        _n(6)
        cu_kv, max_kv, total_kv = ctx.kv_span(d.window)
        return ext().latent_attention(
            h, weight, d.sizes(), d.scale, freq, kv_norm_w, float(eps), kv_proj.weight, kv_proj.offset["uv"], w_ukt, w_uv, pool,
            positions, ctx.slot_mapping, ctx.block_tables, ctx.context_lens, ctx.cu_seqlens_q, cu_kv, ctx.row_seq, ctx.row_ctx,
            int(ctx.max_seqlen_q), int(ctx.max_seqlen_k), max_kv, total_kv, q_norm_w, q_weight, sink, LATENT_IMPL)
    p = ref_linear(h, weight)
    q_in = p[:, d.q:] if d.dq is None else ref_linear(ref.latent_of_queries(p, d, q_norm_w, eps, q_weight.shape[1]), q_weight)
    q = ref.latent_project(p, q_in, d, freq, kv_norm_w, eps, positions, pool, ctx.slot_mapping)
    w, off = kv_proj.weight, kv_proj.offset
    gate = None if d.g is None else p[:, d.g:d.g + d.heads * (1 if d.head_gate else d.vdim)]
    return ref.latent_attention(q, gate, d, w[off["uk"]:off["uk"] + d.heads * d.dim],
                                w[off["uv"]:off["uv"] + d.heads * d.vdim], pool, ctx, sink)


# ------------------------------------------------------------------ attention whose heads mix their scores
TALK_IMPL = 0           # tests: 1 the general kernels also where a tensor-core form exists, 2 the decode form also in prefill


def talking_attention(p, d: TalkDims, freq, talk, eps: float, pool, positions, ctx, out):
    """Rotation (`freq`: rope_turns), norm per head, cache store, attention with scores talk @ scores to `out`.  talk [H, H]
    fp32, to and from; cache rows [keys | values] of all key heads."""
    if out.is_cuda:
        _n(3)
        ext().talking_attention(p, d.sizes(), d.scale, freq, talk, float(eps), pool, positions, ctx.slot_mapping, ctx.block_tables,
                                ctx.context_lens, ctx.cu_seqlens_q, ctx.cu_seqlens_kv, ctx.row_seq, ctx.row_ctx,
                                int(ctx.max_seqlen_q), int(ctx.max_seqlen_k), int(ctx.total_kv), out, TALK_IMPL)
    else:
        ref.talking_attention(p, d, freq, talk, eps, pool, positions, ctx, out)


# ------------------------------------------------------------------ pre-normed layers with parallel sublayers
SMALL_ROWS = 256        # up to this many rows a projection stays fp32 split-K partial sums for its readers


CHUNK_ROWS = 24         # longest run of a batch from which recurrences work in chunks, on finished projections


def project(h, weight, ctx, rows: Optional[int] = None, wide=None):
    """h @ weight[:rows].T for the ops below: a matrix on CPU, an extension object on CUDA (for up to SMALL_ROWS rows its
    fp32 partial sums, valid until the next product).  `wide` = (first, count): columns that are kept in fp32."""
    if h.is_cuda:
        _n()
        first, count = wide or (0, 0)
        finish = ctx.is_prefill and int(ctx.max_seqlen_q) >= CHUNK_ROWS
        return ext().project(h, weight, int(rows or weight.shape[0]), int(first), int(count), finish)
    return ref_linear(h, weight if rows is None else weight[:rows])


def linear_add_norm(a, weight, x, norm_w, eps: float, add: bool = True, experts=None, out=None):
    """x (+)= a @ weight.T + the mixed outputs of `experts` in fp32, in place; returns RMSNorm(x) * norm_w (norm_w None: x
    itself) in the model's dtype, in `out` if given."""
    if a.is_cuda:
        _n(2)
        y, row_of, mix = experts or (None, None, None)
        return ext().linear_add_norm(a, weight, x, norm_w, float(eps), bool(add), y, row_of, mix, out)
    h = ref.add_norm(ref_linear(a, weight), x, add, norm_w, eps, experts)
    return h if out is None else out.copy_(h)


def glu(p, gate: int, up: int, width: int, spec: GluSpec, out):
    """act(gate) * up of a projection, to `out` (its columns past `width` are zeroed)."""
    if out.is_cuda:
        _n()
        ext().glu(p, int(gate), int(up), int(width), spec.code, float(spec.limit), out)
    else:
        out.copy_(ref._pad_to(ref.glu(p[:, gate:gate + width], p[:, up:up + width], spec.act, spec.limit), out.shape[1]))


def linear_glu(h, weight, up: int, width: int, spec: GluSpec, out):
    """The same of the product h @ weight.T, weight = gate rows, then (from row `up`) up rows; prefill sizes run the gate in
    the GEMM's epilogue."""
    if out.is_cuda:
        _n(2)
        ext().linear_glu(h, weight, int(up), int(width), spec.code, float(spec.limit), out)
    else:
        glu(ref_linear(h, weight), 0, up, width, spec, out)


# ------------------------------------------------------------------ several residual streams
def embed_streams(ids, weight, width: int, streams: int, nxt, eps: float):
    """(fp32 streams [T, streams, width], all the row of the table; the next sublayer's input).  `nxt` = (connection, norm
    weight, norm bias), see `linear_mix_norm`."""
    if weight.is_cuda:
        _n()
        return ext().embed_streams(ids, weight, int(width), int(streams), *nxt, float(eps))
    return ref.embed_streams(ids, weight, width, streams, nxt, eps)


def linear_mix_norm(a, weight, x, connection, nxt, eps: float, dtype, experts=None):
    """The streams after a sublayer that returned y = a @ weight.T (a None: none) + the mixed outputs of `experts`, in fp32
    and in place: x_t <- sum_s mix[s, t] x_s + out[t] y; returns what the next sublayer reads, the layer norm of
    sum_s in[s] x_s, in `dtype` (the model's).

    `connection` = [in | out | mix] of this sublayer.  `nxt` = (connection, norm weight, norm bias) of the next one; its
    connection None: the plain sum, after which the streams are not needed (nor written) any more."""
    if x.is_cuda:
        _n(2)
        y, row_of, mix = experts or (None, None, None)
        return ext().linear_mix_norm(a, weight, x, connection, *nxt, float(eps), y, row_of, mix)
    y = ref_linear(a, weight) if a is not None else None
    return ref.mix_norm(y, x, connection, nxt, eps, dtype, experts)


# ------------------------------------------------------------------ experts
def route_by_table(ids, table, experts: int, ctx):
    """Which rows every expert gets when a token's id names its experts (table [vocab, top], int32).  CPU: [T, top]."""
    if ids.is_cuda:
        _n()
        return ext().route_by_table(ids, table, int(experts), None if ctx.is_prefill else ctx.context_lens)
    return table[ids].long()


def route_by_score(h, weight, correction, top: int, groups: int, keep: int, ctx):
    """Which rows every expert gets, and the weights [T, top], from scores sigmoid(h @ weight.T): see
    `reference_hybrid.route_by_score`.  CPU: ([T, top], weights)."""
    if h.is_cuda:
        _n(3)
        row_of, plan, mix = ext().route_by_score(h, weight, correction, int(top), int(groups), int(keep),
                                                 None if ctx.is_prefill else ctx.context_lens)
        return (row_of, plan), mix
    return ref.route_by_score(ref_linear(h, weight), correction, top, groups, keep)


def route_by_logit(h, weight, bias, top: int, shared: bool, ctx):
    """Which rows every expert gets, their weights [T, top], the softmax of the chosen logits h @ weight.T + bias, and (shared)
    the factor of a shared expert, the sigmoid of the row of `weight` behind the experts'.  CPU: ([T, top], weights, factor)."""
    if h.is_cuda:
        _n(3)
        row_of, plan, mix, factor = ext().route_by_logit(h, weight, bias, int(top), bool(shared),
                                                         None if ctx.is_prefill else ctx.context_lens)
        return (row_of, plan), mix, factor
    return ref.route_by_logit(ref_linear(h, weight), bias, top, shared)


def experts(h, route, weights, w_gate_up, w_down, ff: int, spec: GluSpec):
    """Expert outputs for `linear_add_norm`: every token's chosen experts, mixed there with `weights` [T, top] fp32 (None:
    equal ones).  w_gate_up [E, 2 * padded ff, K]: gate rows, then up rows; w_down [E, N, padded ff]."""
    if h.is_cuda:
        _n(4)
        row_of, plan = route
        return ext().experts(h, plan, row_of.shape[1], w_gate_up, w_down, int(ff), spec.code, float(spec.limit)), row_of, weights
    return ref.experts(h, route, weights, w_gate_up, w_down, ff, spec.act, spec.limit)


# ------------------------------------------------------------------ windowed attention
ATTN_IMPL = 0           # tests: 1 the general kernel also where a tensor-core form exists


def rope_turns(base: float, dims: int, scaling: Optional[dict] = None):
    """Rotation frequencies in turns per position, float64.  `scaling` (factor, original, fast, slow): YaRN; pairs that turn
    less than `slow` times over the `original` positions are slowed down by `factor`, those that turn more than `fast` times
    stay, with a ramp between."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2 * i / max(1, dims)) / (2 * math.pi)
    if scaling:
        def pair(turns):
            return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(pair(scaling["fast"])), 0), min(math.ceil(pair(scaling["slow"])), dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        f = f / scaling["factor"] * ramp + f * (1 - ramp)
    return f


def rope_size(scaling: Optional[dict]) -> float:
    """Factor of cos and sin that goes with `scaling`."""
    return 0.1 * math.log(scaling["factor"]) + 1.0 if scaling else 1.0


def windowed_attention(p, d: WindowDims, freq, q_norm, k_norm, sink, eps: float, k_rows, v_rows, positions, ctx, out,
                       bias=None):
    """Bias, norm over the whole projection, rotation (`freq`: rope_turns), cache store, attention (with a sink, an output
    gate) to `out`.  `bias`: of the packed projection, by column."""
    if out.is_cuda:
        _n(2)
        ext().windowed_attention(p, d.sizes(), d.scale, d.softcap, d.rot_size, freq, bias, q_norm, k_norm, sink, float(eps),
                                 k_rows, v_rows, positions, ctx.slot_mapping, ctx.block_tables, ctx.context_lens,
                                 ctx.cu_seqlens_q, ctx.row_seq, ctx.row_ctx, int(ctx.max_seqlen_q), int(ctx.max_seqlen_k),
                                 out, ATTN_IMPL)
    else:
        ref.windowed_attention(p, d, freq, q_norm, k_norm, sink, eps, k_rows, v_rows, positions, ctx, out, bias)


# ------------------------------------------------------------------ real-gated linear recurrent unit
LRU_IMPL = 0            # tests: 1 the general kernels also where a tensor-core form exists


def real_gated_lru(h, weight, bias, d: LruDims, conv_w, conv_b, gate_w, gate_b, lam, cache, ctx):
    """Projections, convolution, gates and recurrence of a batch of runs up to the output projection.  gate_w [2, blocks, n, n]
    and gate_b [2, channels]: the gate of the decay, then the gate of the input."""
    if h.is_cuda:
        _n(4)
        return ext().real_gated_lru(h, weight, bias, [d.channels, d.blocks, d.y, d.x], d.sharpness, conv_w, conv_b, gate_w,
                                    gate_b, lam, cache.conv_state, cache.state, *_run_args(ctx), ctx.row_seq, LRU_IMPL)
    return ref.real_gated_lru(ref_linear(h, weight, bias), d, conv_w, conv_b, gate_w, gate_b, lam, cache.conv_state,
                              cache.state, ctx)


# ------------------------------------------------------------------ matrix memory
def matrix_memory(p, d: MatrixMemoryDims, i_bias, f_bias, norm_w, eps: float, cache, ctx, out):
    """mLSTM of a batch of runs with head norm and output gate, to `out`."""
    if out.is_cuda:
        _n(3)
        ext().matrix_memory(p, [d.heads, d.dim, d.vdim, d.q, d.k, d.v, d.g, d.i, d.f], d.cap, d.floor, i_bias, f_bias,
                            norm_w, float(eps), cache.state, cache.norm_state, cache.max_state, *_run_args(ctx), out)
    else:
        ref.matrix_memory(p, d, i_bias, f_bias, norm_w, eps, cache.state, cache.norm_state, cache.max_state, ctx, out)
