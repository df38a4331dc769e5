"""Small random Darusun models for the tests."""
import torch

import darusun_oracle as oracle
from bagedra_models import PAGE, engine, errors, feed, save, tokens  # noqa: F401  (drivers that do not depend on the model)


def talking(heads=6, kv_heads=3, dim=20, vdim=28, rot=12, base=5e3, scale=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=rot),
             scale=1.5 * dim ** -0.5 if scale is None else scale)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def latent(heads=5, dim=18, rot=10, vdim=14, rank=26, q_rank=22, window=21, base=3e3, scale=None):
    return "latent_attention", dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, q_rank=q_rank, mask=dict(size=window),
                                    rot=dict(base=base, dims=rot), scale=(dim + rot) ** -0.5 if scale is None else scale)


def dense(ff=56):
    return dict(kind="dense", ff=ff)


def moe(experts=6, top=2, ff=40, shared=36):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top), shared=dict(ff=shared))


def config(layers, width=72, vocab=110, eps=1e-5, mult=0.6):
    """layers: (mixer, feed-forward or None) pairs."""
    return dict(architecture="Darusun", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=mult,
                layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in layers])


def weights(cfg, seed=0, decisive=False):
    """Random tensors by checkpoint name (values exact in bf16).  Attention is peaked, heads mix with either sign, sinks compete
    with the keys.  `decisive`: the biases alone choose the experts, so that no 16-bit run decides a close call differently (the
    weights still vary)."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def put(name, *shape, scale=None, mean=0.0):
        s = shape[-1] ** -0.5 if scale is None else scale
        out[name] = (torch.randn(shape, generator=g) * s + mean).bfloat16().float()

    def gated(p, F):
        for n, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
            put(p + n, *shape)

    put("embed", V, W, scale=0.8)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, D, VD = m["heads"], m["dim"], m["vdim"]
        put(f"l{i}.norm1", scale=0.2, mean=1.0)
        put(p + "o", W, H * VD)
        if layer["type"] == "attention":
            put(p + "q", H * D, W)
            if "kv_from" not in m:
                put(p + "k", m["kv_heads"] * D, W)
                put(p + "v", m["kv_heads"] * VD, W)
            out[p + "talk"] = (0.7 * torch.eye(H) + 0.5 * H ** -0.5 * torch.randn(H, H, generator=g)).bfloat16().float()
        else:
            R, K, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            put(p + "dq", Q, W)
            put(p + "dq.norm", Q, scale=0.2, mean=1.0)
            put(p + "uq", H * (D + R), Q, scale=2 * Q ** -0.5)
            put(p + "dkv", K + R, W)
            put(p + "dkv.norm", K, scale=0.2, mean=1.0)
            put(p + "uk", H * D, K)
            put(p + "uv", H * VD, K)
            put(p + "sink", H, scale=1.0, mean=2.0)
            put(p + "g", H, W)
        mlp, p = layer["mlp"], f"l{i}.mlp."
        if mlp is None:
            continue
        put(f"l{i}.norm2", scale=0.2, mean=1.0)
        if mlp["kind"] == "dense":
            put(p + "up", mlp["ff"], W, scale=1.5 * W ** -0.5)
            put(p + "down", W, mlp["ff"])
            put(p + "act", 2, scale=0.8)
            continue
        E = mlp["router"]["experts"]
        for e in range(E):
            gated(f"{p}e{e}.", mlp["expert"]["ff"])
        put(p + "router", E, W, scale=(0.3 if decisive else 2) * W ** -0.5)
        put(p + "router.b", E, scale=0.7)
        if decisive:
            out[p + "router.b"] = 2.5 * torch.randperm(E, generator=g).float()
        gated(p + "shared.", mlp["shared"]["ff"])
        put(p + "shared.sg", 1, W)
    put("final.norm", scale=0.2, mean=1.0)
    put("head", V, W)
    return out


def pointer_model(spec, at, n, vocab=60, width=48, seed=2, strength=12.0):
    """One attention layer whose token 1 asks for token 0: (cfg, weights, prompt) with token 0 only at place `at` and token 1
    last.  The score (`strength` where the key is seen) lies in dimensions that are not rotated, so that only the mask decides."""
    kind, m = spec
    cfg = config([(spec, None)], width=width, vocab=vocab, mult=4.0)
    w = weights(cfg, seed=seed)
    eps, H, D, p = cfg["norm"]["eps"], m["heads"], m["dim"], "l0.mix."
    e0, e1 = w["embed"][0], w["embed"][1]
    unit = e1 / e1.pow(2).sum()
    if kind == "attention":
        R = m["rot"]["dims"]
        assert R < D
        k0 = (w[p + "k"] @ e0).view(m["kv_heads"], D).repeat_interleave(H // m["kv_heads"], 0).clone()
        k0[:, :R] = 0
        w[p + "q"] = (0.02 * w[p + "q"] + torch.outer(k0.reshape(-1), unit)).bfloat16().float()
        w[p + "talk"] = (torch.eye(H) + 0.1 * w[p + "talk"]).bfloat16().float()
        m["scale"] = 2 * strength / D
    else:
        c0 = oracle.rms(w[p + "dkv"][:m["kv_rank"]] @ e0, eps) * w[p + "dkv.norm"]
        k0 = (w[p + "uk"] @ c0).view(H, D)
        c1 = oracle.rms(w[p + "dq"] @ e1, eps) * w[p + "dq.norm"]
        uq = 0.02 * w[p + "uq"].view(H, D + m["rot_dim"], -1)
        uq[:, :D] += (strength / m["scale"] * k0 / k0.pow(2).sum(-1, keepdim=True))[:, :, None] * (c1 / c1.pow(2).sum())
        w[p + "uq"] = uq.reshape(H * (D + m["rot_dim"]), -1).bfloat16().float()
    prompt = [2 + t % (vocab - 2) for t in tokens(n, 10 ** 6, seed)]
    prompt[at], prompt[-1] = 0, 1
    return cfg, w, prompt


def expected(cfg, w, prompts):
    return {i: oracle.forward(cfg, w, t)[0] for i, t in prompts.items()}
