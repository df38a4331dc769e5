"""Plain, slow statements of the Darusun mechanisms (float64 by default), one function per mechanism.

They take whole sequences, keep no cache and share no code with the package: the tests compare the engine,
its caches and its kernels with them.  Shapes: `x`, `h` [T, width]; weights as stored, [out, in].
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def angles(positions, rot):
    """cos and sin [T, 1, dims / 2] of position * base^(-2 i / dims)."""
    n = rot["dims"]
    f = torch.tensor([rot["base"] ** (-2 * i / n) for i in range(n // 2)], dtype=torch.float64)
    a = positions.to(torch.float64)[:, None, None] * f
    return a.cos(), a.sin()


def rotate_half(x, positions, rot):
    """x [T, heads, D]: entry i below dims / 2 turns with entry i + dims / 2."""
    half = rot["dims"] // 2
    c, s = (t.to(x.dtype) for t in angles(positions, rot))
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def rotate_pairs(x, positions, rot):
    """x [T, heads, D]: entries 2i and 2i + 1 turn together."""
    n = rot["dims"]
    c, s = (t.to(x.dtype) for t in angles(positions, rot))
    out = x.clone()
    for i in range(n // 2):
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c[..., i] - v * s[..., i]
        out[..., 2 * i + 1] = v * c[..., i] + u * s[..., i]
    return out


def softmax(s, seen, sink=None):
    """Over the last axis of s [H, T, T] where `seen`; exp(sink [H]) counts once in the denominator."""
    s = s.masked_fill(~seen, float("-inf"))
    top = s.amax(-1, keepdim=True)
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink[:, None, None] - top)
    return e / total


# ------------------------------------------------------------------ talking-heads attention
def attention_rows(h, w, m, eps):
    """Keys [T, G, D] (rotated, then unit root mean square) and values [T, G, V]."""
    T, G, D, V = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = rotate_half((h @ w["k"].T).view(T, G, D), torch.arange(T), m["rot"])
    return rms(k, eps), (h @ w["v"].T).view(T, G, V)


def mix_heads(s, talk):
    """Raw scores [H, T, T] -> scores: every head gets its own sum over all heads."""
    return torch.stack([sum(talk[h, g] * s[g] for g in range(s.shape[0])) for h in range(s.shape[0])])


def attention(h, w, m, eps, rows):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k, v = (t.repeat_interleave(H // G, 1) for t in rows)
    q = rms(rotate_half((h @ w["q"].T).view(T, H, D), torch.arange(T), m["rot"]), eps)
    s = mix_heads(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], w["talk"])
    p = softmax(s, torch.ones(T, T, dtype=torch.bool).tril())
    return torch.einsum("hij,jhd->ihd", p, v).reshape(T, H * V) @ w["o"].T


# ------------------------------------------------------------------ latent attention
def sliding_window(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def latent_attention(h, w, m, eps):
    T, H, D, R, V, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = ((rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T).view(T, H, D + R)
    y = h @ w["dkv"].T
    c = rms(y[:, :K], eps) * w["dkv.norm"]
    r = rotate_pairs(y[:, None, K:], pos, m["rot"])[:, 0]
    k, v = (c @ w["uk"].T).view(T, H, D), (c @ w["uv"].T).view(T, H, V)
    s = torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihd,jd->hij", rotate_pairs(q[..., D:], pos, m["rot"]), r)
    p = softmax(s * m["scale"], sliding_window(T, m["mask"]["size"]), w["sink"])
    o = torch.einsum("hij,jhd->ihd", p, v) * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w["o"].T


# ------------------------------------------------------------------ feed-forward
def xielu(z, p, q):
    a, b = softplus(p), 0.5 + softplus(q)
    neg = z.clamp(max=0)
    return torch.where(z > 0, a * z * z, b * (torch.exp(neg) - 1 - neg)) + z / 2


def dense_ff(h, w, mlp):
    return xielu(h @ w["up"].T, w["act"][0], w["act"][1]) @ w["down"].T


def expert(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def route(z, top):
    """Router logits z [E] of one token -> {expert: weight}: the softmax over the `top` largest."""
    chosen = sorted(range(len(z)), key=lambda e: -float(z[e]))[:top]
    m = max(float(z[e]) for e in chosen)
    x = {e: math.exp(float(z[e]) - m) for e in chosen}
    return {e: v / sum(x.values()) for e, v in x.items()}


def experts(h, w, mlp):
    out = expert(h, w, "shared.") * sigmoid(h @ w["shared.sg"].T)
    z = h @ w["router"].T + w["router.b"]
    for t in range(h.shape[0]):
        for e, weight in route(z[t], mlp["router"]["top"]).items():
            out[t] += weight * expert(h[t], w, f"e{e}.")
    return out


# ------------------------------------------------------------------ model
def _part(weights, prefix):
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    rows, stream = {}, []
    for i, layer in enumerate(cfg["layers"]):
        mix, mw = layer["mixer"], _part(w, f"l{i}.mix.")
        if layer["type"] == "attention":
            src = mix.get("kv_from")
            if src is None:
                rows[i] = attention_rows(x, mw, mix, eps)
            y = attention(x, mw, mix, eps, rows[i if src is None else src])
        else:
            assert layer["type"] == "latent_attention"
            y = latent_attention(x, mw, mix, eps)
        x = x + m * rms(y, eps) * w[f"l{i}.norm1"]
        mlp = layer.get("mlp")
        if mlp is not None:
            y = {"dense": dense_ff, "moe": experts}[mlp["kind"]](x, _part(w, f"l{i}.mlp."), mlp)
            x = x + m * rms(y, eps) * w[f"l{i}.norm2"]
        stream.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T, torch.stack(stream)
