"""Plain, slow statements of the Bagedra mechanisms (float64 by default), one function per mechanism.

They take whole sequences, keep no cache and share no code with the package: the tests compare the engine,
its caches and its kernels with them.  Shapes: `x`, `h` [T, width]; weights as stored, [out, in].
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def rotate_half(x, positions, dims, base):
    """x [T, ..., D]: the first `dims` entries of the last axis are rotated by position, the rest pass."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    a = positions.to(torch.float64)[:, None] * base ** (-2 * i / dims)
    a = a.reshape(a.shape[0], *([1] * (x.dim() - 2)), dims // 2).to(x.dtype)
    u, v, rest = x[..., :dims // 2], x[..., dims // 2:dims], x[..., dims:]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), rest], -1)


def causal_conv(x, w):
    """x [T, C], w [C, taps]; the last column of w meets the current token, zeros before the start."""
    taps = w.shape[1]
    T = x.shape[0]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


def latent_rows(h, w, m, eps):
    """The rows a latent-attention cache holds: (normed latent [T, kv_rank], rotated shared key part [T, rot_dim])."""
    y = h @ w["dkv"].T
    c = rms(y[:, :m["kv_rank"]], eps) * w["dkv.norm"]
    r = rotate_half(y[:, m["kv_rank"]:], torch.arange(h.shape[0]), m["rot"]["dims"], m["rot"]["base"])
    return c, r


def latent_attention(h, w, m, eps, rows=None):
    T, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = latent_rows(h, w, m, eps) if rows is None else rows
    q = (h @ w["q"].T).view(T, H, D + R)
    qn, qr = q[..., :D], rotate_half(q[..., D:], torch.arange(T), m["rot"]["dims"], m["rot"]["base"])
    kn = (c @ w["uk"].T).view(T, H, D)
    v = (c @ w["uv"].T).view(T, H, V)
    s = (torch.einsum("ihd,jhd->hij", qn, kn) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v).reshape(T, H * V)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def gla_scan(q, k, v, alpha):
    """q, k, alpha [T, H, D], v [T, H, V] -> o [T, H, V], token by token."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def gla(h, w, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w["k"].T).view(T, H, D)
    v = (h @ w["v"].T).view(T, H, V)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    alpha = torch.sigmoid(z).pow(1 / m["tau"]).view(T, H, D)
    o = rms(gla_scan(q, k, v, alpha), eps) * w["norm"]
    return (o.reshape(T, H * V) * silu(h @ w["g"].T)) @ w["o"].T


def delta_scan(q, k, v, g, beta):
    """q, k [T, H, D], v [T, H, V], g, beta [T, H] -> o [T, H, V], token by token."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def unit(x):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def delta(h, w, m, eps):
    T, H, K, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in "qkv")
    q = unit(q.view(T, K, D)) * D ** -0.5
    k = unit(k.view(T, K, D))
    q, k = (x.repeat_interleave(H // K, dim=1) for x in (q, k))
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = rms(delta_scan(q, k, v.view(T, H, V), g, beta), eps) * w["norm"]
    return (o.reshape(T, H * V) * silu(h @ w["g"].T)) @ w["o"].T


def dense_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def _part(weights, prefix):
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    rows, stream = {}, []
    for i, layer in enumerate(cfg["layers"]):
        m, mw = layer["mixer"], _part(w, f"l{i}.mix.")
        kind = layer["type"]
        if kind == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                rows[i] = latent_rows(x, mw, m, eps)
            y = latent_attention(x, mw, m, eps, rows[i if src is None else src])
        else:
            y = {"gla": gla, "delta": delta}[kind](x, mw, m, eps)
        x = x + rms(y, eps) * w[f"l{i}.norm1"]
        if layer.get("mlp") is not None:
            x = x + rms(dense_ff(x, _part(w, f"l{i}.mlp.")), eps) * w[f"l{i}.norm2"]
        stream.append(x)
    return rms(x, eps) * w["final.norm"] @ w["head"].T, torch.stack(stream)
