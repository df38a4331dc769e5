"""Plain PyTorch statements of the ops of hybrid models: norms on a 32-bit residual, short convolution, gated linear
attention, gated delta rule, matrix memory, real-gated recurrence, paged latent attention, attention with mixed heads, windowed
and chunked attention, experts, several residual streams.

Like `reference.py`: the execution path on CPU tensors.  A batch is a concatenation of runs of rows, one run per
request, with the request's state slot and the position of its first row; a run that starts at position 0 starts
from a zero state.
"""
from __future__ import annotations

import math
from typing import List, Optional, Tuple

import torch
import torch.nn.functional as F

from .reference import _rotate


def runs(ctx) -> List[Tuple[int, int, int, int, int]]:
    """(request, first row, end row, position of the first row, state slot) of every run of the batch."""
    lens = ctx.context_lens.tolist()
    cu = list(range(len(lens) + 1)) if ctx.cu_seqlens_q is None else ctx.cu_seqlens_q.tolist()
    slots = ctx.state_slots.tolist() if ctx.state_slots is not None else [-1] * len(lens)
    return [(i, cu[i], cu[i + 1], n - (cu[i + 1] - cu[i]), slots[i]) for i, n in enumerate(lens)
            if n > 0 and cu[i + 1] > cu[i]]


def _pad_to(x: torch.Tensor, width: int) -> torch.Tensor:
    return F.pad(x, (0, width - x.shape[-1]))


def _rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


# ------------------------------------------------------------------ residual stream
def embed_scaled(ids, weight, width: int, scale: float):
    h = F.embedding(ids, weight)
    x = h[:, :width].float() * scale
    return x, _pad_to(x.to(weight.dtype), weight.shape[1])


def post_norm_add(y, x, weight, eps: float, experts=None, factor=None):
    s = y[:, : x.shape[1]].float()
    if factor is not None:
        s = s * factor[:, None]
    if experts is not None:
        s = s + experts[:, : x.shape[1]].float()
    x += _rms(s, eps) * weight
    return _pad_to(x.to(y.dtype), y.shape[1])


def xielu(z, coef):
    """coef[0] z^2 + z / 2 above 0, coef[1] (exp(z) - 1 - z) + z / 2 below."""
    n = z.clamp(max=0)
    return torch.where(z > 0, coef[0] * z * z, coef[1] * (torch.expm1(n) - n)) + z / 2


def rms_norm_wide(x, weight, eps: float, width: int, dtype):
    return _pad_to((_rms(x, eps) * weight).to(dtype), width)


def gelu_tanh_and_mul(gu, up_off: int, width: int):
    a = F.gelu(gu[:, :width].float(), approximate="tanh") * gu[:, up_off:up_off + width].float()
    return _pad_to(a.to(gu.dtype), -(-width // 8) * 8)


# ------------------------------------------------------------------ recurrent layers
def short_conv(p, conv_w, conv_state, ctx):
    """silu(depthwise causal convolution) of the first C columns of p, per run; updates the kept inputs."""
    return F.silu(causal_conv(p[:, :conv_w.shape[0]].float(), conv_w, conv_state, ctx))


def causal_conv(x, conv_w, conv_state, ctx):
    """Depthwise causal convolution of x [T, C] fp32, per run; updates the kept inputs."""
    C, taps = conv_w.shape
    out = torch.zeros_like(x)
    for _, lo, hi, start, slot in runs(ctx):
        past = x.new_zeros(taps - 1, C) if start == 0 else conv_state[slot]
        seq = torch.cat([past, x[lo:hi]])
        out[lo:hi] = sum(seq[j:j + hi - lo] * conv_w[:, j] for j in range(taps))
        if taps > 1:
            conv_state[slot] = seq[hi - lo:]
    return out


def gated_head_norm(o, gate, norm_w, eps: float, dtype):
    """rms(o) * norm_w * silu(gate) per head; o [T, H, V] fp32 -> [T, pad8(H * V)]."""
    T, H, V = o.shape
    y = (_rms(o, eps) * norm_w).reshape(T, H * V) * F.silu(gate.float())
    return _pad_to(y.to(dtype), -(-H * V // 8) * 8)


def gla(p, z, d, z_bias, norm_w, eps: float, state, ctx):
    """d: sizes and column offsets (`ops.hybrid.GlaDims`); p packed projections, z decay projection [T, H * D]."""
    T, H, D, V = p.shape[0], d.heads, d.dim, d.vdim
    q = p[:, d.q:d.q + H * D].float().view(T, H, D) * D ** -0.5
    k = p[:, d.k:d.k + H * D].float().view(T, H, D)
    v = p[:, d.v:d.v + H * V].float().view(T, H, V)
    alpha = torch.exp(F.logsigmoid(z[:, : H * D].float() + z_bias) / d.tau).view(T, H, D)
    o = q.new_zeros(T, H, V)
    for _, lo, hi, start, slot in runs(ctx):
        S = state.new_zeros(H, D, V) if start == 0 else state[slot].clone()
        for t in range(lo, hi):
            S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        state[slot] = S
    return gated_head_norm(o, p[:, d.g:d.g + H * V], norm_w, eps, p.dtype)


def delta_rule(p, d, conv_w, a_log, dt_bias, norm_w, eps: float, conv_state, state, ctx):
    """d: `ops.hybrid.DeltaDims`; p packed projections whose first columns are q | k | v."""
    T, H, K, D, V = p.shape[0], d.heads, d.kv_heads, d.dim, d.vdim
    c = short_conv(p, conv_w, conv_state, ctx)
    q, k = c[:, : K * D].reshape(T, K, D), c[:, K * D: 2 * K * D].reshape(T, K, D)
    q, k = (x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + d.unit_eps) for x in (q, k))
    q, k = (x.repeat_interleave(H // K, 1) for x in (q * D ** -0.5, k))
    v = c[:, 2 * K * D:].to(p.dtype).float().view(T, H, V)
    beta = torch.sigmoid(p[:, d.b:d.b + H].float())
    g = torch.exp(-torch.exp(a_log) * F.softplus(p[:, d.a:d.a + H].float() + dt_bias))
    o = q.new_zeros(T, H, V)
    for _, lo, hi, start, slot in runs(ctx):
        S = state.new_zeros(H, D, V) if start == 0 else state[slot].clone()
        for t in range(lo, hi):
            S = g[t][:, None, None] * S
            u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        state[slot] = S
    return gated_head_norm(o, p[:, d.g:d.g + H * V], norm_w, eps, p.dtype)


def real_gated_lru(p, d, conv_w, conv_b, gate_w, gate_b, lam, conv_state, state, ctx):
    """d: `ops.hybrid.LruDims`; p packed projections with their biases.  S <- a S + sqrt(1 - a^2) i u per channel with
    log a = -sharpness r softplus(lam); u = convolution of the x branch, r and i its block-diagonal gates; the y branch
    multiplies the output."""
    C, n = d.channels, d.channels // d.blocks
    u = (causal_conv(p[:, d.x:d.x + C].float(), conv_w, conv_state, ctx) + conv_b).to(p.dtype).float()
    z = torch.einsum("tbk,gbnk->gtbn", u.view(-1, d.blocks, n), gate_w.float()).reshape(2, -1, C)
    r, i = torch.sigmoid(z + gate_b[:, None])
    log_a = -d.sharpness * r * F.softplus(lam)
    a, write = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * u
    o = torch.zeros_like(u)
    for _, lo, hi, start, slot in runs(ctx):
        S = state.new_zeros(C) if start == 0 else state[slot].clone()
        for t in range(lo, hi):
            S = a[t] * S + write[t]
            o[t] = S
        state[slot] = S
    y = o * F.gelu(p[:, d.y:d.y + C].float(), approximate="tanh")
    return _pad_to(y.to(p.dtype), -(-C // 8) * 8)


# ------------------------------------------------------------------ latent attention
def latent_of_queries(p, d, norm_w, eps: float, width: int):
    c = _rms(p[:, d.dq:d.dq + d.q_rank].float(), eps) * norm_w
    return _pad_to(c.to(p.dtype), width)


def latent_project(p, q_in, d, turns, norm_w, eps: float, positions, pool, slots):
    """Writes the cache rows (normed latent | rotated shared key part) of a layer that owns a cache and returns the
    queries (first columns of `q_in`) with their rotated part rotated, [T, H, dim + rot]."""
    T = p.shape[0]

    def turned(x):
        return rope_rows(x, positions, turns, d.rot_dims, d.half, 1.0).to(x.dtype)

    q = q_in[:, :d.heads * (d.dim + d.rot)].reshape(T, d.heads, d.dim + d.rot).clone()
    q[..., d.dim:] = turned(q[..., d.dim:])
    if d.kv is not None:
        kv = p[:, d.kv:d.kv + d.rank + d.rot]
        c = (_rms(kv[:, : d.rank].float(), eps) * norm_w).to(p.dtype)
        r = turned(kv[:, None, d.rank:])[:, 0]
        ok = slots >= 0
        flat = pool.view(-1, pool.shape[-1])
        flat[slots[ok].long(), : d.rank + d.rot] = torch.cat([c, r], -1)[ok].to(pool.dtype)
    return q


def latent_attention(q, gate, d, w_uk, w_uv, pool, ctx, sink=None):
    """Causal attention of the rows of `q` over the cache rows of their requests (inside the window), times sigmoid(gate)."""
    T, H = q.shape[0], d.heads
    out = torch.zeros(T, H, d.vdim, dtype=torch.float32)
    for i, lo, hi, start, _ in runs(ctx):
        n = start + hi - lo
        blocks = ctx.block_tables[i][: -(-n // pool.shape[1])].long()
        rows = pool[blocks].reshape(-1, pool.shape[-1])[:n].float()
        c, r = rows[:, : d.rank], rows[:, d.rank: d.rank + d.rot]
        kn = (c @ w_uk[:, : d.rank].float().T).view(n, H, d.dim)
        v = (c @ w_uv[:, : d.rank].float().T).view(n, H, d.vdim)
        s = torch.einsum("ihd,jhd->hij", q[lo:hi, :, : d.dim].float(), kn)
        s = (s + torch.einsum("ihd,jd->hij", q[lo:hi, :, d.dim:].float(), r)) * d.scale
        at, key = torch.arange(start, n)[:, None], torch.arange(n)[None, :]
        hidden = key > at
        if d.window > 0:
            hidden |= at - key >= d.window
        out[lo:hi] = torch.einsum("hij,jhv->ihv", softmax_with_sink(s.masked_fill(hidden, float("-inf")), sink), v)
    if gate is not None:
        g = torch.sigmoid(gate.float())
        out = out * (g[:, :, None] if d.head_gate else g.view(T, H, d.vdim))
    y = out.reshape(T, H * d.vdim)
    return _pad_to(y.to(q.dtype), -(-H * d.vdim // 8) * 8)


def softmax_with_sink(s, sink):
    """Softmax of s [H, i, j] over j whose denominator also holds exp(sink [H]) (None: not)."""
    if sink is None:
        return torch.softmax(s, -1)
    n = s.shape[-1]
    return torch.softmax(torch.cat([s, sink[:, None, None].expand(-1, s.shape[1], 1)], -1), -1)[..., :n]


# ------------------------------------------------------------------ attention whose heads mix their scores
def talking_attention(p, d, turns, talk, eps: float, pool, positions, ctx, out):
    """Stores the batch's keys and values in the pages (layers that own them) and writes attention to `out`.  d:
    `ops.hybrid.TalkDims`."""
    T, H, G, D, V = p.shape[0], d.heads, d.kv_heads, d.dim, d.vdim

    def turned(off, heads):
        x = p[:, off:off + heads * D].reshape(T, heads, D)
        return _rms(rope_rows(x, positions, turns, d.rot_dims, True, 1.0), eps)

    q = turned(d.q, H)
    if d.k is not None:
        ok = ctx.slot_mapping >= 0
        rows = torch.zeros(T, pool.shape[-1])
        rows[:, :G * D] = turned(d.k, G).reshape(T, G * D)
        rows[:, d.v_col:d.v_col + G * V] = p[:, d.v:d.v + G * V].float()
        pool.view(-1, pool.shape[-1])[ctx.slot_mapping[ok].long()] = rows[ok].to(pool.dtype)
    o = torch.zeros(T, H, V)
    for i, lo, hi, start, _ in runs(ctx):
        n = start + hi - lo
        blocks = ctx.block_tables[i][: -(-n // pool.shape[1])].long()
        rows = pool[blocks].reshape(-1, pool.shape[-1])[:n].float()
        k, v = rows[:, :G * D].reshape(n, G, D), rows[:, d.v_col:d.v_col + G * V].reshape(n, G, V)
        s = torch.einsum("ihd,jhd->hij", q[lo:hi], k.repeat_interleave(H // G, 1)) * d.scale
        s = torch.einsum("hg,gij->hij", talk, s)
        hidden = torch.arange(n)[None, :] > torch.arange(start, n)[:, None]
        o[lo:hi] = torch.einsum("hij,jhv->ihv", torch.softmax(s.masked_fill(hidden, float("-inf")), -1),
                                v.repeat_interleave(H // G, 1))
    out.copy_(_pad_to(o.reshape(T, H * V).to(p.dtype), out.shape[1]))


# ------------------------------------------------------------------ pre-normed layers
def add_norm(y, x, add: bool, norm_w, eps: float, experts=None):
    """x (+)= y + the mixed expert outputs, in place; returns rms(x) * norm_w, or x itself where norm_w is None."""
    if not add:
        x.zero_()
    x += y[:, : x.shape[1]].float()
    if experts is not None:
        x += experts[:, : x.shape[1]].float()
    n = x if norm_w is None else _rms(x, eps) * norm_w
    return _pad_to(n.to(y.dtype), y.shape[1])


def embed_streams(ids, weight, width: int, streams: int, nxt, eps: float):
    x = F.embedding(ids, weight)[:, None, :width].float().repeat(1, streams, 1)
    return x, _streams_in(x, nxt, eps, weight.shape[1], weight.dtype)


def _streams_in(x, nxt, eps: float, width: int, dtype):
    c, w, b = nxt
    u = x.sum(1) if c is None else torch.einsum("s,tsw->tw", c[: x.shape[1]], x)
    u = u - u.mean(-1, keepdim=True)
    return _pad_to((_rms(u, eps) * w + b).to(dtype), width)


def mix_norm(y, x, connection, nxt, eps: float, dtype, experts=None):
    """x [T, S, W] after a sublayer (in place) and the next one's input; connection [in (S) | out (S) | mix (S * S, from * S +
    to)]."""
    S, W = x.shape[1:]
    width = (y if y is not None else experts).shape[1]
    total = sum(t[:, :W].float() for t in (y, experts) if t is not None)
    out, mix = connection[S:2 * S], connection[2 * S:].view(S, S)
    x.copy_(torch.einsum("st,nsw->ntw", mix, x) + out[:, None] * total[:, None])
    return _streams_in(x, nxt, eps, width, dtype)


def glu(gate, up, act: str, limit: float):
    """act(gate) * up ("silu"), or the clamped form ("clamped"): g * sigmoid(1.702 g) * (u + 1) with g = min(gate, limit)
    and u = up clamped to +-limit."""
    g, u = gate.float(), up.float()
    if act == "silu":
        return (F.silu(g) * u).to(gate.dtype)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)).to(gate.dtype)


def route_by_score(z, correction, top: int, groups: int, keep: int):
    """Chosen experts [T, top] and their weights: of the `keep` groups (equal, of neighbours) whose two largest choice scores
    sigmoid(z) + correction have the largest sums, the `top` experts with the largest choice scores; weights are the
    scores without correction over their sum."""
    T, E = z.shape[0], correction.numel()
    s = torch.sigmoid(z[:, :E].float())
    choice = (s + correction).view(T, groups, -1)
    best = choice.topk(min(2, choice.shape[2]), -1).values.sum(-1).topk(keep, -1).indices
    out = torch.ones(T, groups, dtype=torch.bool).scatter(1, best, False)
    ids = choice.masked_fill(out[..., None], float("-inf")).view(T, E).topk(top, -1).indices
    w = s.gather(1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def route_by_logit(z, bias, top: int, shared: bool):
    """Chosen experts [T, top] (largest logits z + bias), the softmax of their logits, and the sigmoid of the column of z behind
    the experts' (or None)."""
    E = bias.numel()
    best = (z[:, :E].float() + bias).topk(top, -1)
    return best.indices, torch.softmax(best.values, -1), torch.sigmoid(z[:, E].float()) if shared else None


def experts(h, ids, weights, w_gate_up, w_down, ff: int, act: str, limit: float):
    """Sum over a token's experts `ids` [T, top] of weight * down(glu(gate, up)); weights None: equal ones."""
    out = torch.zeros(h.shape[0], w_down.shape[1], dtype=torch.float32, device=h.device)
    half = w_gate_up.shape[1] // 2
    for e in ids.unique().tolist():
        t, j = (ids == e).nonzero(as_tuple=True)
        gu = h[t].float() @ w_gate_up[e].float().T
        y = _pad_to(glu(gu[:, :ff], gu[:, half:half + ff], act, limit).to(h.dtype), w_down.shape[2]).float() @ w_down[e].float().T
        out.index_add_(0, t, y * (1.0 / ids.shape[1] if weights is None else weights[t, j][:, None]))
    return out


def rope_rows(x, positions, turns, dims: int, half: bool, size: float):
    """Rotation of the first `dims` columns of x [T, H, D] by position * turns: columns 2i and 2i + 1 together, or (half) i
    and i + dims / 2; cos and sin times `size`."""
    a = 2 * math.pi * positions.double()[:, None, None] * turns
    c, s = (size * a.cos()).float(), (size * a.sin()).float()
    x = x.float()
    if half:
        return torch.cat([_rotate(x[..., :dims], c, s), x[..., dims:]], -1)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], -1)


def windowed_attention(p, d, turns, q_norm, k_norm, sink, eps: float, k_rows, v_rows, positions, ctx, out, bias=None):
    """Stores the batch's keys and values in the pages and writes attention (times sigmoid(gate)) to `out`.
    d: `ops.hybrid.WindowDims`."""
    T, H, G, D, V = p.shape[0], d.heads, d.kv_heads, d.dim, d.value_dim
    if bias is not None:
        p = p + bias
    q, k = p[:, d.q:d.q + H * D].float(), p[:, d.k:d.k + G * D]
    v = k if d.v is None else p[:, d.v:d.v + G * V]
    rope = positions, turns, d.rot_dims, d.half, d.rot_size
    q = rope_rows((_rms(q, eps) * q_norm).view(T, H, D), *rope).to(p.dtype)
    kn = rope_rows((_rms(k.float(), eps) * k_norm).view(T, G, D), *rope)
    ok = ctx.slot_mapping >= 0
    slots = ctx.slot_mapping[ok].long()
    bs = k_rows.shape[2]
    k_rows[slots // bs, :, slots % bs, :D] = kn[ok].to(k_rows.dtype)
    v_rows[slots // bs, :, slots % bs, :V] = v.reshape(T, G, V)[ok].to(v_rows.dtype)
    o = torch.zeros(T, H, V)
    for i, lo, hi, start, _ in runs(ctx):
        n = start + hi - lo
        blocks = ctx.block_tables[i][: -(-n // bs)].long()
        ks, vs = (r[blocks][..., :w].transpose(1, 2).reshape(-1, G, w)[:n].float().repeat_interleave(H // G, 1)
                  for r, w in ((k_rows, D), (v_rows, V)))
        s = torch.einsum("ihd,jhd->hij", q[lo:hi].float(), ks) * d.scale
        if d.softcap:
            s = d.softcap * torch.tanh(s / d.softcap)
        at, key = torch.arange(start, n)[:, None], torch.arange(n)[None, :]
        hidden = key > at
        if d.window > 0:
            hidden |= at - key >= d.window
        if d.chunk > 0:
            hidden |= key < at // d.chunk * d.chunk
        o[lo:hi] = torch.einsum("hij,jhd->ihd", softmax_with_sink(s.masked_fill(hidden, float("-inf")), sink), vs)
    y = o.reshape(T, H * V)
    if d.g is not None:
        y = y * torch.sigmoid(p[:, d.g:d.g + H * V].float())
    out.copy_(_pad_to(y.to(p.dtype), out.shape[1]))


def matrix_memory(p, d, i_bias, f_bias, norm_w, eps: float, state, norm_state, max_state, ctx, out):
    """d: `ops.hybrid.MatrixMemoryDims`; p packed projections."""
    T, H, D, V = p.shape[0], d.heads, d.dim, d.vdim
    q = p[:, d.q:d.q + H * D].float().view(T, H, D) * D ** -0.5
    k = p[:, d.k:d.k + H * D].float().view(T, H, D)
    v = p[:, d.v:d.v + H * V].float().view(T, H, V)
    gi = d.cap * torch.tanh((p[:, d.i:d.i + H].float() + i_bias) / d.cap)
    gf = F.logsigmoid(d.cap * torch.tanh((p[:, d.f:d.f + H].float() + f_bias) / d.cap))
    o = q.new_zeros(T, H, V)
    for _, lo, hi, start, slot in runs(ctx):
        if start == 0:
            S, n, m = state.new_zeros(H, D, V), state.new_zeros(H, D), state.new_zeros(H)
        else:
            S, n, m = state[slot].clone(), norm_state[slot].clone(), max_state[slot].clone()
        for t in range(lo, hi):
            top = torch.maximum(gf[t] + m, gi[t])
            keep, write = torch.exp(gf[t] + m - top), torch.exp(gi[t] - top)
            m = top
            S = keep[:, None, None] * S + (write[:, None] * k[t])[:, :, None] * v[t][:, None, :]
            n = keep[:, None] * n + write[:, None] * k[t]
            den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + d.floor
            o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
        state[slot], norm_state[slot], max_state[slot] = S, n, m
    y = _rms(o, eps).reshape(T, H * V) * norm_w * torch.sigmoid(p[:, d.g:d.g + H * V].float())
    out.copy_(_pad_to(y.to(p.dtype), out.shape[1]))
