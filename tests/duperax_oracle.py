"""Plain, slow statements of the Duperax mechanisms (float64 by default), one function per mechanism.

They take whole sequences, keep no cache and share no code with the package: the tests compare the engine,
its caches and its kernels with them.  Shapes: `h` [T, width]; weights as stored, [out, in].
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * weight + bias


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------ streams
def streams_in(x, w):
    """What a sublayer reads of the streams x [T, S, width]."""
    return sum(w["in"][s] * x[:, s] for s in range(x.shape[1]))


def streams_out(x, y, w):
    """The streams after a sublayer that returned y; mix[from, to]."""
    S = x.shape[1]
    return torch.stack([sum(w["mix"][s, t] * x[:, s] for s in range(S)) + w["out"][t] * y for t in range(S)], 1)


# ------------------------------------------------------------------ attention
def rope_frequencies(rot):
    """(angle per position of every pair, factor of cos and sin)."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    if not s:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def dim(turns):
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim(s["fast"])), 0), min(math.ceil(dim(s["slow"])), n - 1)
    for i in range(n // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        f[i] = f[i] / s["factor"] * ramp + f[i] * (1 - ramp)
    return torch.tensor(f, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1


def rotate_half(x, positions, rot):
    """x [T, heads, D]: entry i below dims / 2 turns with entry i + dims / 2."""
    half = rot["dims"] // 2
    f, size = rope_frequencies(rot)
    a = positions.to(torch.float64)[:, None] * f
    c, s = (size * a.cos()).to(x.dtype)[:, None], (size * a.sin()).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def sliding_window(i, j, size):
    return (i - j >= 0) & (i - j < size)


def chunks(i, j, size):
    return (j <= i) & (i // size == j // size)


def attention(h, w, m, eps, visible, rotated):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[n].T + w.get(n + ".b", 0) for n in "qkv")
    pos = torch.arange(T)
    q = (rms(q, eps) * w["q.norm"]).view(T, H, D)
    k = (rms(k, eps) * w["k.norm"]).view(T, G, D)
    if rotated:
        q, k = rotate_half(q, pos, m["rot"]), rotate_half(k, pos, m["rot"])
    k, v = (t.repeat_interleave(H // G, 1) for t in (k, v.view(T, G, V)))
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    if rotated:
        s = m["softcap"] * torch.tanh(s / m["softcap"])
    s = s.masked_fill(~visible(pos[:, None], pos[None, :], m["mask"]["size"]), float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v).reshape(T, H * V) @ w["o"].T


# ------------------------------------------------------------------ real-gated linear recurrent unit
def causal_conv(x, w, bias):
    T, taps = x.shape[0], w.shape[1]
    past = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(past[j:j + T] * w[:, j] for j in range(taps)) + bias


def block_linear(u, w, b):
    """w [blocks, n, n], b [blocks, n] on the equal parts of u."""
    n = w.shape[1]
    return torch.cat([u[:, i * n:(i + 1) * n] @ w[i].T + b[i] for i in range(w.shape[0])], -1)


def lru_scan(u, r, i, lam):
    """u, gates r and i [T, C] -> states [T, C], token by token."""
    state, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        a = torch.exp(-8 * r[t] * torch.logaddexp(lam, torch.zeros_like(lam)))
        state = a * state + torch.sqrt(1 - a * a) * i[t] * u[t]
        out.append(state)
    return torch.stack(out)


def rglru(h, w, m, eps):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    r, i = (sigmoid(block_linear(u, w[n], w[n + ".b"])) for n in ("ra", "ri"))
    return (lru_scan(u, r, i, w["lam"]) * y) @ w["o"].T


# ------------------------------------------------------------------ feed-forward
def dense_ff(h, w, mlp):
    L = mlp["limit"]
    g, u = (h @ w["gate"].T).clamp(max=L), (h @ w["up"].T).clamp(-L, L)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w["down"].T


def route(z, correction, router):
    """Router logits z [E] of one token -> {expert: weight}."""
    E, top = router["experts"], router["top"]
    n, keep = router["groups"]["count"], router["groups"]["keep"]
    s = sigmoid(z)
    choice = (s + correction).tolist()
    size = E // n
    score = [sum(sorted(choice[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(n)]
    best = sorted(range(n), key=lambda g: -score[g])[:keep]
    allowed = [e for e in range(E) if e // size in best]
    chosen = sorted(allowed, key=lambda e: -choice[e])[:top]
    total = sum(s[e] for e in chosen) + 1e-20
    return {e: s[e] / total for e in chosen}


def experts(h, w, mlp):
    out = torch.zeros_like(h)
    z = h @ w["router"].T
    for t in range(h.shape[0]):
        for e, weight in route(z[t], w["correction"], mlp["router"]).items():
            y = silu(w[f"e{e}.gate"] @ h[t]) * (w[f"e{e}.up"] @ h[t])
            out[t] += weight * (w[f"e{e}.down"] @ y)
    return out


# ------------------------------------------------------------------ model
def _part(weights, prefix):
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


def mixer(kind, h, w, m, eps):
    if kind == "rglru":
        return rglru(h, w, m, eps)
    if kind == "attention":
        return attention(h, w, m, eps, sliding_window, False)
    assert kind == "attention_2", kind
    return attention(h, w, m, eps, chunks, True)


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits [T, vocab] and the sum of the streams after every layer run [runs, T, width]."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)][:, None].repeat(1, cfg["streams"], 1)
    trace = []
    for i in layer_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        hc = _part(w, p + "hc1.")
        h = layer_norm(streams_in(x, hc), w[p + "norm1"], w[p + "norm1.b"], eps)
        x = streams_out(x, mixer(layer["type"], h, _part(w, p + "mix."), layer["mixer"], eps), hc)
        mlp = layer.get("mlp")
        if mlp is not None:
            hc = _part(w, p + "hc2.")
            h = layer_norm(streams_in(x, hc), w[p + "norm2"], w[p + "norm2.b"], eps)
            x = streams_out(x, {"dense": dense_ff, "moe": experts}[mlp["kind"]](h, _part(w, p + "mlp."), mlp), hc)
        trace.append(x.sum(1))
    h = layer_norm(x.sum(1), w["final.norm"], w["final.norm.b"], eps)
    return h @ w["head"].T * cfg["logit_scale"], torch.stack(trace)
