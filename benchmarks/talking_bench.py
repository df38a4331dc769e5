"""Darusun beside the dense decoder: the model of the layer throughput and the kernel table (see hybrid_bench.py).

    python bench.py --layers darusun [--small]
    python benchmarks/talking_bench.py          # the kernels as a readable table
"""
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

WINDOW, EXPERTS, TOP, RANK, ROT, MULT = 1024, 16, 2, 512, 64, 0.5


def key_heads(heads):
    return max(2, heads // 16)


def model_config(width, heads, ff, rank=RANK):
    """Eight layers, every second attention layer on another one's rows, half with experts.  Feed-forwards use as many weights
    per token as the dense decoder's: xIELU has two matrices, the experts of a token share the rest with the shared one."""
    talk = dict(heads=heads, kv_heads=key_heads(heads), dim=128, vdim=128, scale=128 ** -0.5, rot=dict(base=1e6, dims=64))
    lat = dict(heads=heads, dim=128, rot_dim=ROT, vdim=128, kv_rank=rank, q_rank=3 * width // 8, mask=dict(size=WINDOW),
               rot=dict(base=1e4, dims=ROT), scale=192 ** -0.5)
    dense = dict(kind="dense", ff=3 * ff // 2)
    moe = dict(kind="moe", expert=dict(ff=ff // (2 * TOP)), router=dict(experts=EXPERTS, top=TOP), shared=dict(ff=ff // 2))
    layers = []
    for i in range(0, 8, 4):
        layers += [dict(type="attention", mixer=talk, mlp=dense), dict(type="latent_attention", mixer=lat, mlp=moe),
                   dict(type="attention", mixer=dict(talk, kv_from=i), mlp=moe), dict(type="latent_attention", mixer=lat, mlp=dense)]
    return dict(architecture="Darusun", vocab=32768, width=width, norm=dict(eps=1e-6), residual_mult=MULT, layers=layers)


def kernel_table(only=""):
    """Kernels at width 4096, 32 heads, and the like kernels of the dense decoder."""
    from benchmarks.hybrid_bench import DECODE, PREFILL, compare, graphed
    from benchmarks.kernel_bench import peaks, timeit
    from fastcache_b200 import ops
    from fastcache_b200.ops import hybrid
    from fastcache_b200.ops.loader import ext
    from fastcache_b200.utils.context import Context
    hbm, tf, src = peaks()
    e = ext()
    dev, bf = "cuda", torch.bfloat16
    W, H, GD, FF, D, V, R = 4096, 32, 8, 12288, 128, 128, ROT
    rows = []

    def rnd(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev, dtype=torch.float32) * scale).to(dtype)

    def i32(*v):
        return torch.tensor(v, dtype=torch.int32, device=dev)

    def add(kernel, case, fn, byts, flops=0.0, like=None, like_case=None):
        if only and only not in kernel and "(dense)" not in kernel:
            return
        ms = timeit(graphed(fn))
        roof = max(byts / (hbm * 1e9), flops / (tf * 1e12)) * 1e3
        rows.append({"kernel": kernel, "case": case, "ms": round(ms, 4), "of_roofline": round(roof / ms, 3), "like": like,
                     "like_case": like_case or case})

    T = 8192
    none = torch.empty(0, device=dev, dtype=bf)
    y = rnd(T, W)
    # ---- norms on the residual stream
    for t in (T, 64):
        x, res, wbf, w32 = rnd(t, W, dtype=torch.float32), rnd(t, W), torch.ones(W, device=dev, dtype=bf), torch.ones(W, device=dev)
        yt, case = y[:t].contiguous(), f"{t} rows"
        add("add_rms_norm (dense)", case, lambda: e.add_rms_norm(yt, res, wbf, 1e-6), t * W * 2 * 4)
        add("norm + add", case, lambda: e.linear_post_norm_add(yt, none, None, x, w32, 1e-6), t * W * 12, like="add_rms_norm (dense)")
        row_of = torch.randperm(t * TOP, device=dev).int().view(t, TOP)
        mix, factor = torch.rand(t, TOP, device=dev), torch.rand(t, device=dev)
        ey = e.as_projection(rnd(t * TOP, W))
        add("expert mix + norm + add", case, lambda: e.linear_post_norm_add(yt, none, None, x, w32, 1e-6, ey, row_of, mix, factor),
            t * W * (12 + 2 * TOP), like="add_rms_norm (dense)")
        del x, ey, res
    # ---- feed-forwards
    fe, fs, fd = FF // (2 * TOP), FF // 2, 3 * FF // 2
    gu, down = rnd(EXPERTS, 2 * fe, W, scale=0.01), rnd(EXPERTS, W, fe, scale=0.01)
    sgu, sdown = rnd(2 * fs, W, scale=0.01), rnd(W, fs, scale=0.01)
    router, bias = rnd(EXPERTS + 8, W, scale=W ** -0.5), torch.zeros(EXPERTS, device=dev)
    wg, wd = rnd(2 * FF, W, scale=0.01), rnd(W, FF, scale=0.01)
    xu, xd, coef = rnd(fd, W, scale=0.01), rnd(W, fd, scale=0.01), torch.tensor([0.7, 1.2], device=dev)
    act = torch.empty(T, fs, device=dev, dtype=bf)

    def dense_ff(h):
        return ops.linear(ops.linear_silu_mul(h, wg), wd)

    def shared(h):
        a = act[:h.shape[0]]
        hybrid.linear_glu(h, sgu, fs, fs, hybrid.GluSpec(), a)
        return ops.linear(a, sdown)

    for t in (T, 64, 128, 8, 1):
        h, ctx, case = y[:t].contiguous(), Context(is_prefill=True), f"{t} rows"
        route, mix, _ = hybrid.route_by_logit(h, router, bias, TOP, True, ctx)
        first = route[1][:EXPERTS + 1].cpu()
        used = int((first[1:] > first[:-1]).sum())
        flops, like = 2.0 * t * 3 * FF * W, "feed-forward GEMMs (dense)"
        add(like, case, lambda: dense_ff(h), 3 * FF * W * 2 + t * (W + FF) * 4, flops)
        add("xIELU feed-forward", case, lambda: ops.linear(hybrid.linear_xielu(h, xu, coef, fd), xd), 2 * fd * W * 2 + t * (W + fd) * 4, flops,
            like=like)
        add("experts", case, lambda: hybrid.experts(h, route, mix, gu, down, fe, hybrid.GluSpec()),
            used * 3 * W * fe * 2 + t * 2 * W * 4, flops / 2, like=like)
        add("shared expert", case, lambda: shared(h), 3 * W * fs * 2 + t * (W + fs) * 4, flops / 2, like=like)
        add("router: logits, choice, plan", case, lambda: hybrid.route_by_logit(h, router, bias, TOP, True, ctx),
            t * W * 2 + EXPERTS * W * 2)
    del gu, down, wg, wd, act, sgu, sdown, xu, xd
    # ---- attention
    cos_sin = torch.ones(16384, D, device=dev, dtype=torch.float32)
    freq = hybrid.rope_turns(1e6, 64).cuda()
    talk = torch.eye(H, device=dev) + 0.1 * torch.randn(H, H, device=dev)
    sink = torch.zeros(H, device=dev)

    def dense_attention(qkv, pos, slots, kc, vc, bt, lens, cu, n):
        q = ops.rope_qknorm_store(qkv, pos, cos_sin, H, GD, D, None, None, 1e-6, kc, vc, slots)
        if cu is None:
            return ops.decode_attention(q, kc, vc, bt, lens, D ** -0.5)
        return ops.prefill_attention(q, kc, vc, bt, cu, lens, D ** -0.5, n)

    for b, n in PREFILL + [(-b, n) for b, n in DECODE]:
        prefill, b = b > 0, abs(b)
        pages = -(-n // 256)
        bt = torch.arange(b * pages, device=dev, dtype=torch.int32).view(b, -1)
        lens = i32(*([n] * b))
        if prefill:
            pos = torch.arange(n, device=dev).repeat(b)
            seq = torch.arange(b, device=dev, dtype=torch.int32).repeat_interleave(n)
            cu, t = torch.arange(b + 1, device=dev, dtype=torch.int32) * n, b * n
        else:
            pos, seq, cu, t = torch.full((b,), n - 1, device=dev), torch.arange(b, device=dev, dtype=torch.int32), None, b
        slots = (bt[seq.long(), pos // 256] * 256 + (pos % 256).int()).int()
        ctx = (pos + 1).int()
        case, kind = f"{b} x {n}", "prefill" if prefill else "decode"
        full = b * n * (n + 1) / 2 if prefill else b * n
        win = b * (sum(min(i + 1, WINDOW) for i in range(n)) if prefill else min(n, WINDOW))
        like = f"rope + store + {kind} attention (dense)"
        kc, vc, qkv = rnd(b * pages, GD, 256, D), rnd(b * pages, GD, 256, D), rnd(t, (H + 2 * GD) * D)
        add(like, case, lambda: dense_attention(qkv, pos, slots, kc, vc, bt, lens, cu, n),
            t * (2 * H + 2 * GD) * D * 4 + (0 if prefill else b * n * GD * D * 4), full * H * 4 * D)
        q = rnd(t, H, D)
        if prefill:
            add("prefill attention (dense)", case, lambda: ops.prefill_attention(q, kc, vc, bt, cu, lens, D ** -0.5, n),
                t * (2 * H + 2 * GD) * D * 2, full * H * 4 * D)
        else:
            add("decode attention (dense)", case, lambda: ops.decode_attention(q, kc, vc, bt, lens, D ** -0.5), b * n * GD * D * 4,
                full * H * 4 * D)
        del kc, vc, qkv, q
        out = torch.empty(t, H * V, device=dev, dtype=bf)
        for G in (key_heads(H), GD):
            d = hybrid.TalkDims(H, G, D, V, 64, D ** -0.5, 0, H * D, (H + G) * D, G * D)
            pool, p = rnd(b * pages, 256, G * (D + V)), rnd(t, (H + 2 * G) * D)
            pr = e.as_projection(p)
            # least work: scores head by head, the mix, the values
            add(f"store + mixed {kind} attention, {G} key heads", case,
                lambda: e.talking_attention(pr, d.sizes(), d.scale, freq, talk, 1e-6, pool, pos, slots, bt, lens, cu, cu,
                                            seq if prefill else None, ctx if prefill else None, n if prefill else 0, n, b * n, out, 0),
                t * (2 * H + 2 * G) * D * 4 + (0 if prefill else b * n * G * (D + V) * 2), full * (H * 2 * (D + V) + 2 * H * H), like=like)
            del pool, p, pr
        if prefill:
            q, kv, rot = rnd(t, H, D + R), rnd(t, H * (D + V)), rnd(t, R)
            add("windowed latent prefill attention", case,
                lambda: e.latent_prefill_rows(q, kv, rot, None, cu, cu, D, V, 0.07, n, 0, WINDOW, sink),
                t * 2 * (H * (D + R) + H * (D + V) + R + H * V), win * H * 2 * (D + R + V), like="prefill attention (dense)")
            del q, kv, rot
        else:
            pool, qa, hg = rnd(b * pages, 256, RANK + R), rnd(b, H, RANK + R), torch.ones(b, H, device=dev)
            add("windowed absorbed latent attention", case,
                lambda: e.latent_decode_rows(qa, pool, bt, lens, RANK, 0.07, 0, 0, 1, WINDOW, sink, hg), win * (RANK + R) * 2,
                win * H * 2 * (2 * RANK + R), like="decode attention (dense)")
            del pool, qa
    return compare(rows), src


if __name__ == "__main__":
    for r in kernel_table(sys.argv[1] if len(sys.argv) > 1 else "")[0]:
        print(json.dumps(r))
