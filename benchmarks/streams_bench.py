"""Duperax beside the dense decoder: the model of the layer throughput and the kernel table (see hybrid_bench.py).

    python bench.py --layers duperax [--small]
    python benchmarks/streams_bench.py          # the kernels as a readable table
"""
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

WINDOW, CHUNK, CAP, EXPERTS, TOP, GROUPS, KEEP, STREAMS, BLOCK = 1024, 2048, 30.0, 16, 2, 4, 2, 4, 256
SCALING = dict(factor=4.0, original=4096, fast=32.0, slow=1.0)


def model_config(width, heads, ff, _rank=0):
    """Six layers, two of them run twice: eight layer runs, half with experts that use as much per token as a dense layer."""
    size = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5)
    win = ("attention", dict(size, mask=dict(size=WINDOW)))
    chk = ("attention_2", dict(size, mask=dict(size=CHUNK), softcap=CAP, rot=dict(base=1e4, dims=128, scaling=SCALING)))
    lru = ("rglru", dict(width=width, blocks=width // BLOCK, conv=4))
    dense = dict(kind="dense", ff=ff, limit=7.0)
    moe = dict(kind="moe", expert=dict(ff=ff // TOP), router=dict(experts=EXPERTS, top=TOP, groups=dict(count=GROUPS, keep=KEEP)))
    order = [(lru, dense), (win, moe), (lru, moe), (chk, dense), (lru, dense), (chk, moe)]
    return dict(architecture="Duperax", vocab=32768, width=width, streams=STREAMS, logit_scale=1.0, norm=dict(eps=1e-6),
                loop=dict(start=2, stop=4, times=2), layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in order])


def kernel_table():
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
    W, H, G, FF, D, S = 4096, 32, 8, 12288, 128, STREAMS
    rows = []

    def rnd(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev, dtype=torch.float32) * scale).to(dtype)

    def i32(*v):
        return torch.tensor(v, dtype=torch.int32, device=dev)

    def add(kernel, case, fn, byts, flops=0.0, like=None, like_case=None):
        ms = timeit(graphed(fn))
        roof = max(byts / (hbm * 1e9), flops / (tf * 1e12)) * 1e3
        rows.append({"kernel": kernel, "case": case, "ms": round(ms, 4), "of_roofline": round(roof / ms, 3), "like": like,
                     "like_case": like_case or case})

    T = 8192
    f32 = dict(dtype=torch.float32)
    y = rnd(T, W)
    # ---- residual streams
    for t in (T, 64):
        x, res, wbf = rnd(t, S, W, **f32), rnd(t, W), torch.ones(W, device=dev, dtype=bf)
        hc = torch.cat([torch.full((S,), 1.0 / S), torch.ones(S), torch.eye(S).flatten()]).cuda()
        nw, nb, yt, case = torch.ones(W, device=dev), torch.zeros(W, device=dev), y[:t].contiguous(), f"{t} rows"
        add("add_rms_norm (dense)", case, lambda: e.add_rms_norm(yt, res, wbf, 1e-6), t * W * 2 * 4)
        p = e.as_projection(yt)
        add("mix of the streams + norm", case, lambda: e.mix_norm(p, x, hc, hc, nw, nb, 1e-6), t * W * (8 * S + 4),
            like="add_rms_norm (dense)")
        row_of = torch.randperm(t * TOP, device=dev).int().view(t, TOP)
        mix = torch.rand(t, TOP, device=dev)
        ey = e.as_projection(rnd(t * TOP, W))
        add("expert mix + mix of the streams + norm", case,
            lambda: e.linear_mix_norm(None, None, x, hc, hc, nw, nb, 1e-6, ey, row_of, mix), t * W * (8 * S + 2 + 2 * TOP),
            like="add_rms_norm (dense)")
        del x, ey, res
    # ---- feed-forwards
    gu, down = rnd(EXPERTS, FF, W, scale=0.01), rnd(EXPERTS, W, FF // TOP, scale=0.01)
    router, correction = rnd(EXPERTS, W, scale=W ** -0.5), torch.zeros(EXPERTS, device=dev)
    wg, wd = rnd(2 * FF, W, scale=0.01), rnd(W, FF, scale=0.01)

    def dense_ff(h):
        return ops.linear(ops.linear_silu_mul(h, wg), wd)

    act = torch.empty(T, FF, device=dev, dtype=bf)

    def clamped_ff(h, out):
        hybrid.linear_glu(h, wg, FF, FF, hybrid.GluSpec("clamped", 7.0), out)
        return ops.linear(out, wd)

    for t in (T, 64, 128, 8, 1):
        h, ctx, case = y[:t].contiguous(), Context(is_prefill=True), f"{t} rows"
        route, mix = hybrid.route_by_score(h, router, correction, TOP, GROUPS, KEEP, ctx)
        first = route[1][:EXPERTS + 1].cpu()
        used = int((first[1:] > first[:-1]).sum())
        flops = 2.0 * t * 3 * FF * W
        ff_bytes = 3 * FF * W * 2 + t * (W + FF) * 4
        add("feed-forward GEMMs (dense)", case, lambda: dense_ff(h), ff_bytes, flops)
        add("clamped feed-forward", case, lambda: clamped_ff(h, act[:t]), ff_bytes, flops, like="feed-forward GEMMs (dense)")
        add("experts", case, lambda: hybrid.experts(h, route, mix, gu, down, FF // TOP, hybrid.GluSpec()),
            used * 3 * W * (FF // TOP) * 2 + t * 2 * W * 4, flops, like="feed-forward GEMMs (dense)")
        add("router: scores, choice, plan", case, lambda: hybrid.route_by_score(h, router, correction, TOP, GROUPS, KEEP, ctx),
            t * W * 2 + EXPERTS * W * 2)
    del gu, down, wg, wd, act
    # ---- attention (bias, norms, rotation, store, attention)
    kinds = {"windowed": hybrid.WindowDims(H, G, D, 0, D ** -0.5, WINDOW, 0, H * D, None, (H + G) * D, D),
             "chunked, capped": hybrid.WindowDims(H, G, D, D, D ** -0.5, 0, 0, H * D, None, (H + G) * D, D, CHUNK, CAP, True,
                                                  hybrid.rope_size(SCALING))}
    freqs = {"windowed": torch.empty(0, dtype=torch.float64, device=dev), "chunked, capped": hybrid.rope_turns(1e4, D, SCALING).cuda()}
    qn, kn = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
    cos_sin = torch.ones(16384, D, device=dev, dtype=torch.float32)

    def dense_attention(qkv, pos, slots, kc, vc, bt, lens, cu, n):
        q = ops.rope_qknorm_store(qkv, pos, cos_sin, H, G, D, None, None, 1e-6, kc, vc, slots)
        if cu is None:
            return ops.decode_attention(q, kc, vc, bt, lens, D ** -0.5)
        return ops.prefill_attention(q, kc, vc, bt, cu, lens, D ** -0.5, n)

    for b, n in PREFILL + [(-b, n) for b, n in DECODE]:
        prefill, b = b > 0, abs(b)
        pages = -(-n // 256)
        bt = torch.arange(b * pages, device=dev, dtype=torch.int32).view(b, -1)
        kc, vc = rnd(b * pages, G, 256, D), rnd(b * pages, G, 256, D)
        lens = i32(*([n] * b))
        if prefill:
            pos = torch.arange(n, device=dev).repeat(b)
            seq = torch.arange(b, device=dev, dtype=torch.int32).repeat_interleave(n)
            cu, t = torch.arange(b + 1, device=dev, dtype=torch.int32) * n, b * n
        else:
            pos, seq, cu, t = torch.full((b,), n - 1, device=dev), torch.arange(b, device=dev, dtype=torch.int32), None, b
        slots = (bt[seq.long(), pos // 256] * 256 + (pos % 256).int()).int()
        case = f"{b} x {n}"
        kind = "prefill" if prefill else "decode"
        qkv, bias = rnd(t, (H + 2 * G) * D), rnd((H + 2 * G) * D)
        io = t * (2 * H + 2 * G) * D * 2 * 2
        kv = 0 if prefill else G * D * 4
        full = b * n * (n + 1) / 2 if prefill else b * n
        add(f"rope + store + {kind} attention (dense)", case,
            lambda: dense_attention(qkv, pos, slots, kc, vc, bt, lens, cu, n), io + b * n * kv, full * H * 4 * D)
        pr = e.as_projection(qkv)
        out = torch.empty(t, H * D, device=dev, dtype=bf)
        ctx = (pos + 1).int()
        for name, d in kinds.items():
            def see(i):
                return min(i + 1, WINDOW) if d.window else i % CHUNK + 1
            seen = b * (sum(see(i) for i in range(n)) if prefill else see(n - 1))
            add(f"norms + store + {name} {kind} attention", case,
                lambda: e.windowed_attention(pr, d.sizes(), d.scale, d.softcap, d.rot_size, freqs[name], bias if d.chunk else None, qn, kn,
                                             None, 1e-6, kc, vc, pos, slots, bt, lens, cu, seq if prefill else None,
                                             ctx if prefill else None, n if prefill else 0, 0, out, 0),
                io + b * see(n - 1) * kv, seen * H * 4 * D, like=f"rope + store + {kind} attention (dense)")
        del kc, vc, qkv
    # ---- recurrent unit (projections excluded) beside the gated linear attention of another hybrid model
    gd = [H, D, D, 16, 0, H * D, 2 * H * D, 3 * H * D, 4 * H * D]
    proj = rnd(T, 4 * H * D + 16)
    none = torch.empty(0, device=dev, dtype=bf)
    a2, zb, hn = rnd(H * D, 16, scale=0.3), torch.ones(H * D, device=dev), torch.ones(D, device=dev)
    C, taps, blocks = W, 4, W // BLOCK
    xy, bias = rnd(T, 2 * C), rnd(2 * C, scale=0.1)
    cw, cb, lam = rnd(C, taps, scale=0.5, **f32), torch.zeros(C, device=dev), torch.linspace(-7, -2, C, device=dev)
    gw, gb = rnd(2, blocks, BLOCK, BLOCK, scale=BLOCK ** -0.5), torch.zeros(2, C, device=dev)

    def unit(h, st, cs, cu, lens, slots, n, seq):
        return e.real_gated_lru(h, none, bias, [C, blocks, 0, C], 8.0, cw, cb, gw, gb, lam, cs, st, cu, lens, slots, n, seq, 0)

    for b, n in PREFILL:
        cu = torch.arange(b + 1, device=dev, dtype=torch.int32) * n
        lens, slots = i32(*([n] * b)), torch.arange(b, device=dev, dtype=torch.int32)
        seq = torch.arange(b, device=dev, dtype=torch.int32).repeat_interleave(n)
        fl = b * n * H * 64 * 2 * 2 * D + b * n * H * 4 * D * D
        st = torch.zeros(b, H, D, D, device=dev)
        add("gla chunks (other hybrid model)", f"{b} x {n}", lambda: e.gla(proj, none, a2, zb, hn, 1e-6, st, gd, 16.0, cu, lens, slots, n),
            T * 2 * 6 * H * D, fl)
        s1, cs = torch.zeros(b, C, device=dev), torch.zeros(b, taps - 1, C, device=dev)
        add("recurrent unit: convolution, gates, scan", f"{b} x {n}", lambda: unit(xy, s1, cs, cu, lens, slots, n, seq), T * C * 6,
            T * 4.0 * C * BLOCK, like="gla chunks (other hybrid model)")
    for b, dense in ((64, "64 x 2048"), (128, "128 x 1024"), (8, "8 x 8192"), (1, "1 x 4096")):
        lens, slots = i32(*([100] * b)), torch.arange(b, device=dev, dtype=torch.int32)
        s1, cs, h1 = torch.zeros(b, C, device=dev), torch.zeros(b, taps - 1, C, device=dev), xy[:b].contiguous()
        add("recurrent unit: convolution, step", f"{b} requests", lambda: unit(h1, s1, cs, None, lens, slots, 1, None),
            2 * C * BLOCK * 2 + b * C * (6 + 8 + 8 * (taps - 1)), like="rope + store + decode attention (dense)", like_case=dense)
    return compare(rows), src


if __name__ == "__main__":
    for r in kernel_table()[0]:
        print(json.dumps(r))
