"""Small random Duperax models for the tests."""
import torch

import duperax_oracle as oracle
from bagedra_models import PAGE, engine, errors, feed, tokens  # noqa: F401  (drivers that do not depend on the model)
from lekilix_models import save  # noqa: F401


def attention(heads=6, kv_heads=2, dim=24, vdim=20, window=20, scale=None):
    return "attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window),
                             scale=dim ** -0.5 if scale is None else scale)


def chunked(heads=6, kv_heads=3, dim=20, vdim=28, rot=16, chunk=24, base=5e3, scaling=(8.0, 64, 16.0, 1.5), softcap=12.0, scale=None):
    """scaling: (factor, original, fast, slow)"""
    r = dict(base=base, dims=rot)
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return "attention_2", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=r, mask=dict(size=chunk), softcap=softcap,
                               scale=dim ** -0.5 if scale is None else scale)


def rglru(width=36, blocks=3, taps=4):
    return "rglru", dict(width=width, blocks=blocks, conv=taps)


def dense(ff=56, limit=1.2):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts=6, top=2, ff=40, groups=3, keep=2):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, groups=dict(count=groups, keep=keep)))


def config(layers, width=72, vocab=110, eps=1e-5, streams=3, logit_scale=1.5, loop=None):
    """layers: (mixer, feed-forward or None) pairs; loop: (start, stop, times)."""
    cfg = dict(architecture="Duperax", vocab=vocab, width=width, streams=streams, logit_scale=logit_scale, norm=dict(eps=eps),
               layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in layers])
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def weights(cfg, seed=0, decisive=False):
    """Random tensors by checkpoint name (values exact in bf16).  Attention is peaked, decays range from forgetting to keeping,
    the feed-forward reaches its clamps, choice scores are of either sign, streams mix without growing.  `decisive`: the
    corrections alone choose the experts, so that no 16-bit run decides a close call differently (the weights still vary)."""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    out = {}

    def put(name, *shape, scale=None, mean=0.0):
        s = shape[-1] ** -0.5 if scale is None else scale
        out[name] = (torch.randn(*shape, generator=g) * s + mean).bfloat16().float()

    def norm(name):
        put(name, W, scale=0.2, mean=1.0)
        put(name + ".b", W, scale=0.2)

    put("embed", V, W, scale=1.0)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        for q in (1,) if layer["mlp"] is None else (1, 2):
            norm(f"l{i}.norm{q}")
            put(f"l{i}.hc{q}.in", S, scale=0.4, mean=0.6)
            put(f"l{i}.hc{q}.out", S, scale=0.4, mean=0.6)
            out[f"l{i}.hc{q}.mix"] = (0.8 * torch.eye(S) + 0.25 * torch.randn(S, S, generator=g)).bfloat16().float()
        if layer["type"] == "rglru":
            C, B = m["width"], m["blocks"]
            for n in "yx":
                put(p + n, C, W)
                put(f"{p}{n}.b", C, scale=0.3)
            put(p + "conv", C, m["conv"], scale=0.6)
            put(p + "conv.b", C, scale=0.3)
            for n in ("ra", "ri"):
                put(p + n, B, C // B, C // B, scale=2 * (C // B) ** -0.5)
                put(f"{p}{n}.b", B, C // B, scale=0.5)
            put(p + "lam", C, scale=2.0, mean=-3.0)
            put(p + "o", W, C)
        else:
            H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, size in (("q", H * D), ("k", G * D), ("v", G * VD)):
                put(p + n, size, W)
                if layer["type"] == "attention_2":
                    put(f"{p}{n}.b", size, scale=0.4)
            put(p + "q.norm", H * D, scale=0.3, mean=1.8)
            put(p + "k.norm", G * D, scale=0.2, mean=1.2)
            put(p + "o", W, H * VD)
        mlp, p = layer["mlp"], f"l{i}.mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            for n, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                put(p + n, *shape, scale=None if n == "down" else 1.5 * W ** -0.5)
            continue
        F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
        for e in range(E):
            for n, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                put(f"{p}e{e}.{n}", *shape)
        put(p + "router", E, W, scale=2 * W ** -0.5)
        put(p + "correction", E, scale=0.3, mean=-0.5)
        if decisive:
            out[p + "correction"] = -2.5 * 2.0 ** torch.randperm(E, generator=g).float()      # sums of two differ as well
    norm("final.norm")
    put("head", V, W)
    return out


def pointer_model(spec, at, n, vocab=60, width=48, seed=2, strength=6.0):
    """One attention layer whose token 1 asks for token 0: (cfg, weights, prompt) with token 0 only at place `at` and token
    1 last.  The score lies in dimensions that are not rotated, so that only the mask decides whether the key is seen."""
    cfg = config([(spec, None)], width=width, vocab=vocab)
    w = weights(cfg, seed=seed)
    m, eps = spec[1], cfg["norm"]["eps"]
    H, G, D, R = m["heads"], m["kv_heads"], m["dim"], m.get("rot", {}).get("dims", 0)
    assert R < D
    p = "l0.mix."
    hc = {k: w["l0.hc1." + k] for k in ("in", "out", "mix")}
    x = w["embed"][:2, None].repeat(1, cfg["streams"], 1)
    h = oracle.layer_norm(oracle.streams_in(x, hc), w["l0.norm1"], w["l0.norm1.b"], eps)
    k0 = oracle.rms(w[p + "k"] @ h[0] + w.get(p + "k.b", 0), eps) * w[p + "k.norm"]
    k0 = k0.view(G, D).repeat_interleave(H // G, 0).clone()
    k0[:, :R] = 0
    w[p + "q"] = (0.02 * w[p + "q"] + torch.outer(k0.reshape(-1), h[1] / h[1].pow(2).sum())).bfloat16().float()
    if p + "q.b" in w:
        w[p + "q.b"] *= 0
    w[p + "q.norm"] = torch.full((H * D,), strength)
    w[p + "o"] = (w[p + "o"] * 8).bfloat16().float()
    prompt = [2 + t % (vocab - 2) for t in tokens(n, 10 ** 6, seed)]
    prompt[at], prompt[-1] = 0, 1
    return cfg, w, prompt


def expected(cfg, w, prompts):
    return {i: oracle.forward(cfg, w, t)[0] for i, t in prompts.items()}
