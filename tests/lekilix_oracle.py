"""Plain, slow statements of the Lekilix mechanisms (float64 by default), one function per mechanism.

They take whole sequences, keep no cache and share no code with the package: the tests compare the engine,
its caches and its kernels with them.  Shapes: `x`, `h` [T, width]; weights as stored, [out, in].
"""
import torch


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def rotate_pairs(x, positions, dims, base):
    """x [T, heads, D]: entries 2i and 2i + 1 below `dims` turn together by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def sink_softmax(s, sink):
    """Softmax over the last axis of s [H, T, K] with one more term exp(sink_h) in the denominator."""
    top = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def windowed_attention(h, w, m, eps):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w["q"].T, h @ w["k"].T
    v = k.view(T, G, D)
    pos = torch.arange(T)
    q = rotate_pairs((rms(q, eps) * w["q.norm"]).view(T, H, D), pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_pairs((rms(k, eps) * w["k.norm"]).view(T, G, D), pos, m["rot"]["dims"], m["rot"]["base"])
    k, v = (t.repeat_interleave(H // G, 1) for t in (k, v))
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    back = pos[:, None] - pos[None, :]
    s = s.masked_fill((back < 0) | (back >= m["mask"]["size"]), float("-inf"))
    o = torch.einsum("hij,jhd->ihd", sink_softmax(s, w["sink"]), v).reshape(T, H * D)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def matrix_memory_scan(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, V], log gates i, f [T, H] -> o [T, H, V], token by token."""
    H, D, V = q.shape[1], q.shape[2], v.shape[2]
    S, n, m = q.new_zeros(H, D, V), q.new_zeros(H, D), q.new_zeros(H)
    out = []
    for t in range(q.shape[0]):
        top = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        m = top
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        d = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / d[:, None])
    return torch.stack(out)


def mlstm_gates(h, w, cap):
    """(log input gate, log forget gate) [T, H], both through a soft cap."""
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap)
    return i, -torch.logaddexp(-f, torch.zeros_like(f))


def mlstm(h, w, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w["k"].T).view(T, H, D)
    v = (h @ w["v"].T).view(T, H, V)
    o = rms(matrix_memory_scan(q, k, v, *mlstm_gates(h, w, m["gate_cap"])), eps)
    return (o.reshape(T, H * V) * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def dense_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def clamped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def table_experts(h, tokens, w, mlp):
    """Every token's row of the table names its experts; their outputs count equally."""
    top, limit = mlp["router"]["top"], mlp["expert"]["limit"]
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens.tolist()):
        for e in w["table"][tok].long().tolist():
            y = clamped_glu(w[f"e{e}.gate"] @ h[t], w[f"e{e}.up"] @ h[t], limit)
            out[t] += w[f"e{e}.down"] @ y / top
    return out


def _part(weights, prefix):
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def layer_order(cfg):
    """(layer index, whether a pass of the loop starts here) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for _ in range(times) for i in range(a, b)] +
            [(i, False) for i in range(b, n)])


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits [T, vocab] and the residual stream after every layer run [runs, T, width]."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    tokens = torch.as_tensor(tokens)
    eps = cfg["norm"]["eps"]
    x0 = x = w["embed"][tokens] * cfg["embedding"]["scale"]
    stream = []
    for i, enter in layer_order(cfg):
        layer = cfg["layers"][i]
        if enter:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T
        h = rms(x, eps) * (1 + w[f"l{i}.norm1"])
        mix, ff = _part(w, f"l{i}.mix."), _part(w, f"l{i}.mlp.")
        y = {"attention": windowed_attention, "mlstm": mlstm}[layer["type"]](h, mix, layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = y + (dense_ff(h, ff) if mlp["kind"] == "dense" else table_experts(h, tokens, ff, mlp))
        x = x + y
        stream.append(x)
    return rms(x, eps) * (1 + w["final.norm"]) @ w["head"].T, torch.stack(stream)
