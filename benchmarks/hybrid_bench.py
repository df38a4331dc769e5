"""Layer throughput of the hybrid model (Bagedra) beside the dense decoder (Qwen3) at equal size, and the roofline of
its kernels beside the like kernels of the dense decoder.

    python bench.py --layers [--small]        # throughput and kernels, one JSON line
    python benchmarks/hybrid_bench.py [--kernels]    # the same (or the kernels alone) as a readable table

Random weights.  Throughput: whole forward steps through the engine's prefill and decode steps (CUDA graphs in decode),
CUDA events on the engine's stream, 3 warm-up steps, median; the weights and caches of a step are larger than L2.
Kernels: CUDA events around single operations (replays of a CUDA graph), a 256 MB write between samples to flush L2, median; fractions are of the
measured peaks in MEASURED_PEAKS.json (algorithmic bytes and FLOPs).
"""
import json
import os
import statistics
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

# width, heads, feed-forward, latent size
SIZES = {"2k": (2048, 16, 6144, 512), "4k": (4096, 32, 12288, 512), "6k": (6144, 48, 16384, 512)}
PREFILL = [(4, 2048), (1, 8192)]
DECODE = [(64, 2048), (128, 1024), (8, 8192), (1, 4096)]
LAYERS = 8


def hybrid_config(width, heads, ff, rank):
    rot = {"base": 1e4, "dims": 64}
    latent = dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=rank, rot=rot, scale=192 ** -0.5)
    group = [("delta", dict(heads=heads, kv_heads=heads // 2, dim=128, vdim=128, conv=4)), ("latent_attention", latent),
             ("gla", dict(heads=heads, dim=128, vdim=128, tau=16.0)), ("latent_attention", None)]
    layers = []
    for i in range(LAYERS):
        kind, mixer = group[i % 4]
        mixer = mixer or dict(latent, kv_from=i - 2)
        layers.append(dict(type=kind, mixer=mixer, mlp=dict(kind="dense", ff=ff)))
    return dict(architecture="Bagedra", vocab=32768, width=width, embedding=dict(scale=1.0), norm=dict(eps=1e-6),
                layers=layers)


def dense_config(width, heads, ff, rank):
    return dict(model_type="qwen3", architectures=["Qwen3ForCausalLM"], hidden_size=width, num_hidden_layers=LAYERS,
                num_attention_heads=heads, num_key_value_heads=heads // 4, head_dim=128, intermediate_size=ff,
                vocab_size=32768, rope_theta=1e6, rms_norm_eps=1e-6, max_position_embeddings=16384,
                tie_word_embeddings=False)


def _time_steps(fn, stream, n=10, warmup=3):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    out = []
    for _ in range(n):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        with torch.cuda.stream(stream):
            a.record()
            fn()
            b.record()
        torch.cuda.synchronize()
        out.append(a.elapsed_time(b))
    return statistics.median(out)


def throughput(cfg, steps):
    from fastcache_b200 import LLM
    from fastcache_b200.engine.sequence import Sequence
    page = 256
    pages = max(b * -(-(n + 1) // page) for b, n in PREFILL + DECODE) + 8
    llm = LLM(cfg, kvcache_block_size=page, num_kvcache_blocks=pages, max_model_len=8448, max_num_seqs=128,
              max_num_batched_tokens=16384, prefix_caching=False, tokenizer=False)
    r, bm = llm.model_runner, llm.scheduler.block_manager
    g = torch.Generator().manual_seed(0)
    rows = []

    def requests(b, n):
        seqs = [Sequence(torch.randint(0, 32768, (n,), generator=g).tolist()) for _ in range(b)]
        for s in seqs:
            bm.allocate(s)
        return seqs

    def release(seqs):
        for s in seqs:
            bm.deallocate(s)

    stream = r.main_stream or torch.cuda.current_stream()
    for b, n in PREFILL:
        seqs = requests(b, n)
        # the device work of one prefill step, inputs already on the device
        with torch.cuda.stream(stream):
            ids, pos, _ = r.prepare_prefill(seqs)

        @torch.inference_mode()
        def run():
            with torch.cuda.stream(stream):
                r._forward(ids, pos)
        ms = _time_steps(run, stream, steps)
        rows.append({"phase": "prefill", "requests": b, "tokens": n, "ms": round(ms, 3), "tok_s": round(b * n / ms * 1e3)})
        release(seqs)
    for b, n in DECODE:
        seqs = requests(b, n)
        for i, s in enumerate(seqs):
            s.append_token(7 + 11 * i)                  # different ids: they may choose the experts
            bm.may_append(s)
        with torch.cuda.stream(stream):
            r.run_decode(seqs)
        bucket = r._graph_bucket(b)

        def run():
            with torch.cuda.stream(stream):
                r._replay(bucket)
        ms = _time_steps(run, stream, 2 * steps)
        rows.append({"phase": "decode", "requests": b, "context": n, "ms": round(ms, 4), "tok_s": round(b / ms * 1e3)})
        release(seqs)
    assert r.read_device_status() == 0
    llm.exit()
    del llm, r
    import gc
    gc.collect()
    torch.cuda.empty_cache()
    return rows


def graphed(fn):
    """`fn` as a CUDA-graph replay: what is timed is the device, not the launches from Python."""
    stream = torch.cuda.Stream()
    stream.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(stream):
        for _ in range(2):
            fn()
    stream.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=stream):
        fn()
    return g.replay


def kernel_table():
    """Kernels of the 4k size and the like kernels of the dense decoder."""
    from benchmarks.kernel_bench import peaks, timeit
    from fastcache_b200 import ops
    from fastcache_b200.ops.loader import ext
    hbm, tf, src = peaks()
    e = ext()
    dev, bf = "cuda", torch.bfloat16
    W, H, FF, RANK, R, D, V = 4096, 32, 12288, 512, 64, 128, 128
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

    none = torch.empty(0, device=dev, dtype=bf)
    T = 8192
    x32 = rnd(T, W, dtype=torch.float32)
    y, w32, wbf = rnd(T, W), torch.ones(W, device=dev), torch.ones(W, device=dev, dtype=bf)
    res = rnd(T, W)
    add("add_rms_norm (dense)", "8192 rows", lambda: e.add_rms_norm(y, res, wbf, 1e-6), T * W * 2 * 4)
    add("post_norm_add", "8192 rows", lambda: e.linear_post_norm_add(y, none, None, x32, w32, 1e-6), T * W * 12,
        like="add_rms_norm (dense)")
    gu = rnd(T, 2 * FF)
    add("silu_and_mul (dense)", "8192 rows", lambda: ops.silu_and_mul(gu), T * FF * 6)
    add("gelu_mul", "8192 rows (in the GEMM epilogue at prefill sizes)",
        lambda: e.linear_gelu_mul(gu, none, None, FF, FF), T * FF * 6, like="silu_and_mul (dense)")
    del gu

    # ---- prefill attention
    for b, n in PREFILL:
        cu = torch.arange(b + 1, device=dev, dtype=torch.int32) * n
        pairs = b * n * (n + 1) / 2
        kc, vc = rnd(b * n // 256, 8, 256, D), rnd(b * n // 256, 8, 256, D)
        bt = torch.arange(b * n // 256, device=dev, dtype=torch.int32).view(b, -1)
        lens = i32(*([n] * b))
        q = rnd(b * n, H, D)
        add("prefill_attention (dense)", f"{b} x {n}",
            lambda: ops.prefill_attention(q, kc, vc, bt, cu, lens, D ** -0.5, n), b * n * (2 * H + 16) * D * 2,
            pairs * H * 4 * D)
        q = rnd(b * n, H, D + R)
        kv, rot, gate = rnd(b * n, H * (D + V)), rnd(b * n, R), rnd(b * n, H * V)
        add("latent_prefill", f"{b} x {n}", lambda: e.latent_prefill_rows(q, kv, rot, gate, cu, cu, D, V, 0.07, n),
            b * n * 2 * (H * (D + R) + H * (D + V) + R + 2 * H * V), pairs * H * 2 * (D + R + V),
            like="prefill_attention (dense)")
        del kc, vc, kv, q
    # ---- decode attention
    for b, n in DECODE:
        pages = -(-n // 256)
        bt = torch.arange(b * pages, device=dev, dtype=torch.int32).view(b, -1)
        lens = i32(*([n] * b))
        kc, vc = rnd(b * pages, 8, 256, D), rnd(b * pages, 8, 256, D)
        q = rnd(b, H, D)
        add("decode_attention (dense)", f"{b} x {n}",
            lambda: ops.decode_attention(q, kc, vc, bt, lens, D ** -0.5), b * n * 8 * D * 4, b * n * H * 4 * D)
        pool, qa = rnd(b * pages, 256, RANK + R), rnd(b, H, RANK + R)
        add("latent_decode", f"{b} x {n}", lambda: e.latent_decode_rows(qa, pool, bt, lens, RANK, 0.07),
            b * n * (RANK + R) * 2, b * n * H * 2 * (2 * RANK + R), like="decode_attention (dense)")
        del kc, vc, pool
    # ---- recurrences (projections excluded)
    gd = [H, D, V, 16, 0, H * D, 2 * H * D, 2 * H * D + H * V, 2 * H * D + 2 * H * V]
    proj = rnd(T, 2 * H * D + 2 * H * V + 16)
    a2, zb, hn = rnd(H * D, 16, scale=0.3), torch.ones(H * D, device=dev), torch.ones(V, device=dev)
    dd = [H, H // 2, D, V, H * D + H * V, H * D + 2 * H * V, H * D + 2 * H * V + H]
    dproj = rnd(T, H * D + 2 * H * V + 2 * H)
    C = H * D + H * V
    cw, hv = rnd(C, 4, dtype=torch.float32), torch.zeros(H, device=dev)
    for b, n in PREFILL:
        st, cs = torch.zeros(b, H, D, V, device=dev), torch.zeros(b, 3, C, device=dev)
        cu = torch.arange(b + 1, device=dev, dtype=torch.int32) * n
        lens, slots = i32(*([n] * b)), torch.arange(b, device=dev, dtype=torch.int32)
        seq = torch.arange(b, device=dev, dtype=torch.int32).repeat_interleave(n)
        fl = b * n * H * 64 * 2 * (D + V) + b * n * H * 4 * D * V        # chunk products and state updates
        add("gla: chunked recurrence, gates, head norm", f"{b} x {n}",
            lambda: e.gla(proj, none, a2, zb, hn, 1e-6, st, gd, 16.0, cu, lens, slots, n),
            T * 2 * (3 * H * D + 3 * H * V), fl)
        add("delta: convolution, chunked recurrence, gates, head norm", f"{b} x {n}",
            lambda: e.delta_rule(dproj, none, cw, hv, hv, hn, 1e-6, cs, st, dd, 1e-6, cu, lens, slots, n, seq),
            T * 2 * (H * D + 3 * H * V), fl + b * n * H * 2 * D * V)
    for b, dense in ((64, "64 x 2048"), (8, "8 x 8192"), (1, "1 x 4096")):
        st, cs = torch.zeros(b, H, D, V, device=dev), torch.zeros(b, 3, C, device=dev)
        lens, slots = i32(*([100] * b)), torch.arange(b, device=dev, dtype=torch.int32)
        p1, p2 = proj[:b].contiguous(), dproj[:b].contiguous()
        add("gla step", f"{b} requests",
            lambda: e.gla(p1, none, a2, zb, hn, 1e-6, st, gd, 16.0, None, lens, slots, 1), b * H * D * V * 8,
            like="decode_attention (dense)", like_case=dense)
        add("delta inputs + step", f"{b} requests",
            lambda: e.delta_rule(p2, none, cw, hv, hv, hn, 1e-6, cs, st, dd, 1e-6, None, lens, slots, 1, None),
            b * H * D * V * 8, like="decode_attention (dense)", like_case=dense)
    return compare(rows), src


def compare(rows):
    """Adds to every row that names a like kernel how far that one is from its roofline."""
    by = {(r["kernel"], r["case"]): r["of_roofline"] for r in rows}
    for r in rows:
        if r["like"]:
            ref = by.get((r["like"], r["like_case"])) or next(v for (k, _), v in by.items() if k == r["like"])
            r["like_of_roofline"] = ref
            r["times_as_far"] = round(ref / r["of_roofline"], 2)
        else:
            del r["like"], r["like_case"]
    return rows


def run(steps=5, small=False, kernels=True, model="bagedra"):
    """The result as one dict (see `bench.py --layers`)."""
    make, table = hybrid_config, kernel_table
    if model == "lekilix":
        from benchmarks import prenorm_bench
        make, table = prenorm_bench.model_config, prenorm_bench.kernel_table
    elif model == "duperax":
        from benchmarks import streams_bench
        make, table = streams_bench.model_config, streams_bench.kernel_table
    elif model == "darusun":
        from benchmarks import talking_bench
        make, table = talking_bench.model_config, talking_bench.kernel_table
    sizes = {"2k": SIZES["2k"]} if small else SIZES
    out = {"layers": LAYERS, "sizes": {}}
    for name, size in sizes.items():
        ours, dense = throughput(make(*size), steps), throughput(dense_config(*size), steps)
        for a, b in zip(ours, dense):
            a["dense_ms"], a["dense_tok_s"] = b["ms"], b["tok_s"]
        out["sizes"][name] = {"width": size[0], "heads": size[1], "ff": size[2], "rows": ours}
    if kernels:
        out["kernels"], out["peaks"] = table()
    return out


def main():
    if "--kernels" in sys.argv:
        for r in kernel_table()[0]:
            print(json.dumps(r))
        return
    res = run()
    for name, s in res["sizes"].items():
        for r in s["rows"]:
            print(name, json.dumps(r))
    for r in res.get("kernels", ()):
        print(json.dumps(r))


if __name__ == "__main__":
    main()
