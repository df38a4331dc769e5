"""Small random Bagedra models for the tests, and drivers that feed token ids through the engine."""
import json
import os

import torch

import bagedra_oracle as oracle
from fastcache_b200.engine.replay import TokenReplay
from fastcache_b200.llm import LLM

PAGE = 16


def delta(heads=3, kv_heads=1, dim=24, vdim=40, conv=3):
    return "delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def gla(heads=3, dim=20, vdim=24, tau=8.0):
    return "gla", dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def latent(heads=3, dim=40, rot=16, vdim=56, rank=48, base=1e4, scale=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, rot=dict(base=base, dims=rot),
             scale=scale or (dim + rot) ** -0.5)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention", m


def config(mixers, width=88, ff=72, vocab=150, eps=1e-5, embed_scale=1.5, no_mlp=()):
    layers = [dict(type=t, mixer=m, mlp=None if i in no_mlp else dict(kind="dense", ff=ff))
              for i, (t, m) in enumerate(mixers)]
    return dict(architecture="Bagedra", vocab=vocab, width=width, embedding=dict(scale=embed_scale),
                norm=dict(eps=eps), layers=layers)


def weights(cfg, seed=0, rank=12):
    """Random tensors by checkpoint name (values exact in bf16).  Queries are scaled so that attention is peaked and
    recurrent decays spread from short to long memory."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def put(name, *shape, scale=None, mean=0.0):
        s = shape[-1] ** -0.5 if scale is None else scale
        out[name] = (torch.randn(*shape, generator=g) * s + mean).bfloat16().float()

    put("embed", V, W, scale=0.7)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, D, VD = m["heads"], m["dim"], m["vdim"]
        put(f"l{i}.norm1", W, scale=0.2, mean=0.8)
        put(p + "g", H * VD, W)
        put(p + "o", W, H * VD)
        if layer["type"] == "latent_attention":
            R, K = m["rot_dim"], m["kv_rank"]
            put(p + "q", H * (D + R), W, scale=3 * W ** -0.5)
            if "kv_from" not in m:
                put(p + "dkv", K + R, W)
                put(p + "dkv.norm", K, scale=0.2, mean=1.0)
            put(p + "uk", H * D, K)
            put(p + "uv", H * VD, K)
        else:
            put(p + "norm", VD, scale=0.2, mean=1.0)
            KH = m.get("kv_heads", H)
            put(p + "q", KH * D, W)
            put(p + "k", KH * D, W)
            put(p + "v", H * VD, W)
        if layer["type"] == "gla":
            put(p + "a1", rank, W)
            put(p + "a2", H * D, rank, scale=2 * rank ** -0.5)
            put(p + "a2.b", H * D, scale=2.0, mean=2.0)
        if layer["type"] == "delta":
            for n, c in (("q", KH * D), ("k", KH * D), ("v", H * VD)):
                put(p + n + ".conv", c, m["conv"], scale=0.6)
            put(p + "b", H, W)
            put(p + "a", H, W)
            put(p + "A_log", H, scale=0.7, mean=-1.0)
            put(p + "dt_bias", H, scale=0.7, mean=-1.5)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            put(f"l{i}.norm2", W, scale=0.2, mean=0.8)
            for n, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                put(f"l{i}.mlp.{n}", *shape)
                put(f"l{i}.mlp.{n}.b", shape[0], scale=0.3)
    put("final.norm", W, scale=0.2, mean=1.0)
    put("head", V, W)
    return out


def pointer_model(at, n, spec, seed=2, strength=40.0):
    """A latent layer whose token 1 asks for token 0: (cfg, weights, prompt) with token 0 only at place `at` and token 1
    last.  Removing that one key changes the last logits completely."""
    cfg = config([spec], width=40, ff=24, vocab=60)
    w = weights(cfg, seed=seed)
    m, p = spec[1], "l0.mix."
    e0, e1 = w["embed"][0], w["embed"][1]
    c0 = oracle.rms(w[p + "dkv"][:m["kv_rank"]] @ e0, 1e-6) * w[p + "dkv.norm"]
    k0 = (w[p + "uk"] @ c0).view(m["heads"], m["dim"])
    q = w[p + "q"].view(m["heads"], m["dim"] + m["rot_dim"], -1)
    q *= 0.02
    unit = e1 / e1.pow(2).sum()
    for h in range(m["heads"]):
        q[h, :m["dim"]] += strength * (k0[h] / k0[h].pow(2).sum())[:, None] * unit / m["scale"]
    w[p + "q"] = w[p + "q"].bfloat16().float()
    w[p + "o"] = (w[p + "o"] * 4).bfloat16().float()
    prompt = [2 + t % (cfg["vocab"] - 2) for t in tokens(n, 10 ** 6, seed)]
    prompt[at], prompt[-1] = 0, 1
    return cfg, w, prompt


def save(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    save_file({n: t.bfloat16().contiguous() for n, t in w.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def engine(path, device, dtype, max_tokens=1024, requests=4, page=PAGE, **kw):
    return LLM(path, device=device, dtype=dtype, kvcache_block_size=page, num_kvcache_blocks=-(-max_tokens // page),
               max_model_len=max_tokens, max_num_seqs=requests, tokenizer=False, **kw)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed(llm, prompts, schedule):
    """Runs a schedule, a list of steps of (request name, token count); returns the logits of every position by
    request.  A request ends with its last token."""
    replay = TokenReplay(llm)
    at = {i: 0 for i in prompts}
    got = {i: [] for i in prompts}
    for step in schedule:
        entries, end = [], []
        for i, n in step:
            entries.append({"id": i, "tokens": prompts[i][at[i]:at[i] + n], "want": list(range(n))})
            at[i] += n
            if at[i] >= len(prompts[i]):
                end.append(i)
        rows = replay.step(entries, end)
        for (i, n) in step:
            got[i].append(rows[:n])
            rows = rows[n:]
    assert all(at[i] == len(prompts[i]) for i in prompts)
    llm.scheduler.block_manager.check_invariants([])
    return {i: torch.cat(r) for i, r in got.items()}


def errors(got, want):
    """(largest, mean) rms difference of a position's logits (mean taken off), over the rms of all expected logits."""
    d = got.double() - want.double()
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()
    return float(d.max()), float(d.mean())


def expected(cfg, w, prompts):
    return {i: oracle.forward(cfg, w, t)[0] for i, t in prompts.items()}
