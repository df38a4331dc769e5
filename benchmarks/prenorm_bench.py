"""Lekilix beside the dense decoder: the model of the layer throughput and the kernel table (see hybrid_bench.py).

    python bench.py --layers lekilix [--small]
    python benchmarks/prenorm_bench.py          # the kernels as a readable table
"""
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

WINDOW, EXPERTS, TOP = 1024, 16, 2


def model_config(width, heads, ff, _rank=0):
    """Six layers, two of them run twice: eight layer runs, half with experts that use as much per token as a dense layer."""
    att = ("attention", dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, rot=dict(base=1e4, dims=64),
                             mask=dict(size=WINDOW), scale=128 ** -0.5))
    mem = ("mlstm", dict(heads=heads, dim=128, vdim=128, gate_cap=15.0))
    dense = dict(kind="dense", ff=ff)
    moe = dict(kind="moe", expert=dict(ff=ff // TOP, limit=7.0), router=dict(experts=EXPERTS, top=TOP))
    order = [(mem, dense), (att, moe), (mem, moe), (att, dense), (mem, dense), (att, moe)]
    return dict(architecture="Lekilix", vocab=32768, width=width, embedding=dict(scale=1.0), norm=dict(eps=1e-6),
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
    W, H, G, FF, D, V = 4096, 32, 8, 12288, 128, 128
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
    # ---- norms and products of a prefill step
    x32, nw = rnd(T, W, dtype=torch.float32), torch.ones(W, device=dev)
    y, res, wbf = rnd(T, W), rnd(T, W), torch.ones(W, device=dev, dtype=bf)
    add("add_rms_norm (dense)", "8192 rows", lambda: e.add_rms_norm(y, res, wbf, 1e-6), T * W * 2 * 4)
    add("norm of the stream", "8192 rows", lambda: e.stream_norm(x32, nw, 1e-6, None, None), T * W * 6, like="add_rms_norm (dense)")
    row_of = torch.randperm(T * TOP, device=dev).int().view(T, TOP)
    ey = e.as_projection(rnd(T * TOP, W))
    add("expert mix + norm", "8192 rows", lambda: e.stream_norm(x32, nw, 1e-6, ey, row_of), T * W * (10 + 2 * TOP),
        like="add_rms_norm (dense)")
    del ey, res
    wo = rnd(W, H * V + FF, scale=0.01)
    a = rnd(T, H * V + FF)
    K = H * V + FF
    add("GEMM (dense)", "8192 rows", lambda: ops.linear(a, wo), T * (K + W) * 2 + W * K * 2, 2.0 * T * W * K)
    add("out projections, fp32 stream", "8192 rows", lambda: e.linear_add_norm(a, wo, x32, nw, 1e-6, True, None, None, None, None),
        T * K * 2 + W * K * 2 + T * W * 14, 2.0 * T * W * K, like="GEMM (dense)")
    del a, wo
    N = 4 * H * V + 2 * H
    wi = rnd(N, W, scale=0.01)
    add("in projections, fp32 gates", "8192 rows", lambda: e.project(y, wi, N, N - 2 * H, 2 * H, True), T * (W + N) * 2 + N * W * 2,
        2.0 * T * N * W, like="GEMM (dense)")
    del wi
    # ---- experts
    gu, down = rnd(EXPERTS, FF, W, scale=0.01), rnd(EXPERTS, W, FF // TOP, scale=0.01)
    table = ((torch.arange(32768)[:, None] * TOP + torch.arange(TOP)) % EXPERTS).int().cuda()
    spec = hybrid.GluSpec("clamped", 7.0)
    wg, wd = rnd(2 * FF, W, scale=0.01), rnd(W, FF, scale=0.01)

    def dense_ff(h):
        return ops.linear(ops.linear_silu_mul(h, wg), wd)

    for t, case in ((T, "8192 rows"), (64, "64 rows"), (128, "128 rows"), (8, "8 rows"), (1, "1 rows")):
        ids = torch.randint(0, 32768, (t,), device=dev)
        h = y[:t].contiguous()
        ctx = Context(is_prefill=True)
        route = hybrid.route_by_table(ids, table, EXPERTS, ctx)
        flops = 2.0 * t * 3 * FF * W
        used = len(torch.unique(table[ids].long()))
        byts = used * 3 * W * (FF // TOP) * 2 + t * 2 * W * 4
        add("feed-forward GEMMs (dense)", case, lambda: dense_ff(h), 3 * FF * W * 2 + t * (W + FF) * 4, flops)
        add("experts", case, lambda: hybrid.experts(h, route, None, gu, down, FF // TOP, spec), byts, flops,
            like="feed-forward GEMMs (dense)")
        if t in (T, 64):
            add("routing by table", case, lambda: hybrid.route_by_table(ids, table, EXPERTS, ctx), t * (8 + TOP * 12))
    del gu, down, wg, wd
    # ---- windowed attention (norms, rotation, store, attention, gate)
    cols = hybrid.WindowDims(H, G, D, 64, D ** -0.5, WINDOW, 0, H * D, (H + G) * D).sizes()
    freq = hybrid.rope_turns(1e4, 64).cuda()
    qn, kn, sink = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev), torch.zeros(H, device=dev)
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
        qkv = rnd(t, (H + 2 * G) * D)
        full = b * n * (n + 1) / 2 if prefill else b * n
        seen = b * (sum(min(i + 1, WINDOW) for i in range(n)) if prefill else min(n, WINDOW))
        io = t * (2 * H + 2 * G) * D * 2 * 2
        kv = 0 if prefill else G * D * 4
        add(f"rope + store + {kind} attention (dense)", case,
            lambda: dense_attention(qkv, pos, slots, kc, vc, bt, lens, cu, n), io + b * n * kv, full * H * 4 * D)
        pr = e.as_projection(rnd(t, (2 * H + G) * D))
        out = torch.empty(t, H * D, device=dev, dtype=bf)
        ctx = (pos + 1).int()
        add(f"norms + store + windowed {kind} attention", case,
            lambda: e.windowed_attention(pr, cols, D ** -0.5, 0.0, 1.0, freq, None, qn, kn, sink, 1e-6, kc, vc, pos, slots, bt, lens, cu,
                                         seq if prefill else None, ctx if prefill else None, n if prefill else 0, 0, out, 0),
            io + t * H * D * 2 + b * min(n, WINDOW) * kv, seen * H * 4 * D, like=f"rope + store + {kind} attention (dense)")
        del kc, vc, qkv
    # ---- matrix memory (projections excluded) beside the gated linear attention of the other hybrid model
    gd = [H, D, V, 16, 0, H * D, 2 * H * D, 2 * H * D + H * V, 2 * H * D + 2 * H * V]
    proj = rnd(T, 2 * H * D + 2 * H * V + 16)
    none = torch.empty(0, device=dev, dtype=bf)
    a2, zb, hn = rnd(H * D, 16, scale=0.3), torch.ones(H * D, device=dev), torch.ones(V, device=dev)
    md = [H, D, V, 0, H * D, 2 * H * D, 2 * H * D + H * V, 2 * H * D + 2 * H * V, 2 * H * D + 2 * H * V + H]
    mproj, gates = rnd(T, 2 * H * D + 2 * H * V + 2 * H), rnd(T, 2 * H, dtype=torch.float32)
    hb, mw = torch.ones(H, device=dev), torch.ones(H * V, device=dev)
    out = torch.empty(T, H * V, device=dev, dtype=bf)

    def memory(b):
        return torch.zeros(b, H, D, V, device=dev), torch.zeros(b, H, D, device=dev), torch.zeros(b, H, device=dev)

    for b, n in PREFILL:
        cu = torch.arange(b + 1, device=dev, dtype=torch.int32) * n
        lens, slots = i32(*([n] * b)), torch.arange(b, device=dev, dtype=torch.int32)
        fl = b * n * H * 64 * 2 * (D + V) + b * n * H * 4 * D * V
        byts = T * 2 * (3 * H * D + 3 * H * V)
        st = torch.zeros(b, H, D, V, device=dev)
        add("gla chunks (other hybrid model)", f"{b} x {n}",
            lambda: e.gla(proj, none, a2, zb, hn, 1e-6, st, gd, 16.0, cu, lens, slots, n), byts, fl)
        ms, p = memory(b), e.as_projection(mproj, md[7], gates)
        add("mlstm: gates, chunked recurrence, head norm", f"{b} x {n}",
            lambda: e.matrix_memory(p, md, 15.0, 1e-6, hb, hb, mw, 1e-6, *ms, cu, lens, slots, n, out), byts, fl,
            like="gla chunks (other hybrid model)")
    for b, dense in ((64, "64 x 2048"), (128, "128 x 1024"), (8, "8 x 8192"), (1, "1 x 4096")):
        lens, slots = i32(*([100] * b)), torch.arange(b, device=dev, dtype=torch.int32)
        ms, p, o = memory(b), e.as_projection(mproj[:b].contiguous(), md[7], gates[:b].contiguous()), out[:b]
        add("mlstm step", f"{b} requests",
            lambda: e.matrix_memory(p, md, 15.0, 1e-6, hb, hb, mw, 1e-6, *ms, None, lens, slots, 1, o), b * H * D * (V + 1) * 8,
            like="rope + store + decode attention (dense)", like_case=dense)
    return compare(rows), src


if __name__ == "__main__":
    for r in kernel_table()[0]:
        print(json.dumps(r))
