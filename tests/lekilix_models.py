"""Small random Lekilix models for the tests."""
import json
import os

import torch

import lekilix_oracle as oracle
from bagedra_models import PAGE, engine, errors, feed, tokens  # noqa: F401  (drivers that do not depend on the model)


def attention(heads=6, kv_heads=2, dim=24, rot=12, window=20, base=1e4, scale=None):
    return "attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, rot=dict(base=base, dims=rot),
                             mask=dict(size=window), scale=dim ** -0.5 if scale is None else scale)


def mlstm(heads=3, dim=20, vdim=28, cap=9.0):
    return "mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def dense(ff=56):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=2, ff=40, limit=1.5):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def config(layers, width=72, vocab=110, eps=1e-5, embed_scale=2.5, loop=None):
    """layers: (mixer, feed-forward or None) pairs; loop: (start, stop, times)."""
    cfg = dict(architecture="Lekilix", vocab=vocab, width=width, embedding=dict(scale=embed_scale), norm=dict(eps=eps),
               layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in layers])
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def weights(cfg, seed=0):
    """Random tensors by checkpoint name (values exact in bf16; tables int32).  Attention is peaked with sinks that take a
    visible share, forget gates range from forgetting to keeping, expert inputs reach the clamps."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def put(name, *shape, scale=None, mean=0.0):
        s = shape[-1] ** -0.5 if scale is None else scale
        out[name] = (torch.randn(*shape, generator=g) * s + mean).bfloat16().float()

    put("embed", V, W, scale=0.5)
    if cfg.get("loop"):
        put("loop.in", W, 2 * W)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, D = m["heads"], m["dim"]
        put(f"l{i}.norm1", W, scale=0.2)
        put(p + "q", H * D, W)
        if layer["type"] == "attention":
            G = m["kv_heads"]
            put(p + "k", G * D, W)
            put(p + "q.norm", H * D, scale=0.3, mean=1.6)
            put(p + "k.norm", G * D, scale=0.2, mean=1.2)
            put(p + "sink", H, scale=1.0, mean=1.5)
            put(p + "g", H * D, W)
            put(p + "o", W, H * D)
        else:
            VD = m["vdim"]
            put(p + "k", H * D, W)
            # keys lean towards the queries: a first token whose k.q is near zero has outputs of either sign after the head
            # norm, which no 16-bit run can decide
            out[p + "k"] = (0.7 * out[p + "k"] + 0.7 * out[p + "q"]).bfloat16().float()
            put(p + "v", H * VD, W)
            put(p + "g", H * VD, W)
            put(p + "o", W, H * VD)
            put(p + "norm", H * VD, scale=0.2, mean=1.0)
            put(p + "i", H, W, scale=2 * W ** -0.5)
            put(p + "f", H, W, scale=2 * W ** -0.5)
            put(p + "i.b", H, scale=1.0, mean=-1.0)
            put(p + "f.b", H, scale=1.5, mean=3.0)
        mlp, p = layer["mlp"], f"l{i}.mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            for n, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                put(p + n, *shape)
            continue
        F, E, top = mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"]
        for e in range(E):
            for n, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                put(f"{p}e{e}.{n}", *shape, scale=None if n == "down" else 1.5 * W ** -0.5)
        out[p + "table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(V)]).int()
    put("final.norm", W, scale=0.2)
    put("head", V, W)
    return out


def pointer_model(spec, at, n, vocab=60, width=48, seed=2, strength=6.0):
    """One attention layer whose token 1 asks for token 0: (cfg, weights, prompt) with token 0 only at place `at` and token
    1 last.  The score lies in the dimensions that are not rotated, so that only the window decides whether the key is seen."""
    cfg = config([(spec, None)], width=width, vocab=vocab)
    w = weights(cfg, seed=seed)
    m, eps = spec[1], cfg["norm"]["eps"]
    H, G, D, R = m["heads"], m["kv_heads"], m["dim"], m["rot"]["dims"]
    p = "l0.mix."
    h = [oracle.rms(w["embed"][i] * cfg["embedding"]["scale"], eps) * (1 + w["l0.norm1"]) for i in (0, 1)]
    k0 = (oracle.rms(w[p + "k"] @ h[0], eps) * w[p + "k.norm"]).view(G, D).repeat_interleave(H // G, 0).clone()
    k0[:, :R] = 0
    w[p + "q"] = (0.02 * w[p + "q"] + torch.outer(k0.reshape(-1), h[1] / h[1].pow(2).sum())).bfloat16().float()
    w[p + "q.norm"] = torch.full((H * D,), strength)
    w[p + "sink"] = torch.full((H,), 2.0)
    w[p + "o"] = (w[p + "o"] * 4).bfloat16().float()
    prompt = [2 + t % (vocab - 2) for t in tokens(n, 10 ** 6, seed)]
    prompt[at], prompt[-1] = 0, 1
    return cfg, w, prompt


def save(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    save_file({n: (t if t.dtype == torch.int32 else t.bfloat16()).contiguous() for n, t in w.items()},
              os.path.join(path, "model.safetensors"))
    return str(path)


def expected(cfg, w, prompts):
    return {i: oracle.forward(cfg, w, t)[0] for i, t in prompts.items()}
