"""Duperax on a CUDA device: the engine's kernels in bf16 and fp32 against the plain statements."""
import pytest
import torch

import duperax_models as dm
import duperax_oracle as oracle
from test_duperax_cpu import fill_caches

pytestmark = pytest.mark.gpu

LIMIT = {"bfloat16": 0.2, "float32": 2e-4}            # worst position
MEAN_LIMIT = {"bfloat16": 0.03, "float32": 2e-5}      # all positions

# sizes for the tensor-core forms and sizes that only the general kernels take
MODELS = {
    "general": dict(layers=[(dm.rglru(), dm.dense()), (dm.attention(), dm.moe()), (dm.rglru(width=48, blocks=2, taps=2), dm.moe()),
                            (dm.chunked(chunk=70), None)], loop=(1, 3, 2)),
    "odd": dict(layers=[(dm.attention(heads=5, kv_heads=1, dim=13, vdim=22, window=37), dm.moe(experts=3, top=1, ff=11, groups=3, keep=1)),
                        (dm.rglru(width=21, blocks=3, taps=5), dm.dense(45)), (dm.rglru(width=14, blocks=1, taps=1), None),
                        (dm.chunked(heads=2, kv_heads=2, dim=150, vdim=140, rot=150, chunk=64), None)],
                width=61, vocab=77, loop=(0, 2, 2), streams=5),
    "wide": dict(layers=[(dm.attention(heads=4, kv_heads=2, dim=128, vdim=128, window=100), dm.dense(384)),
                         (dm.rglru(width=256, blocks=2, taps=4), dm.moe(experts=8, top=2, ff=128, groups=4, keep=2)),
                         (dm.chunked(heads=8, kv_heads=1, dim=64, vdim=64, rot=64, chunk=128), dm.moe(experts=4, top=2, ff=256, groups=1, keep=1)),
                         (dm.rglru(width=384, blocks=2, taps=4), dm.dense(256))], width=256, vocab=520, loop=(2, 4, 2), streams=2),
    "mid": dict(layers=[(dm.chunked(heads=6, kv_heads=3, dim=112, vdim=80, rot=48, chunk=300), dm.dense(96)),
                        (dm.rglru(width=160, blocks=5, taps=3), dm.moe(experts=16, top=4, ff=64, groups=4, keep=2))], width=128, vocab=200,
                streams=4),
    "many heads": dict(layers=[(dm.attention(heads=36, kv_heads=2, dim=32, vdim=24, window=90), None),
                               (dm.rglru(width=96, blocks=6, taps=2), dm.dense(128))], width=192, vocab=100, loop=(0, 1, 3), streams=1),
}
SINGLE = {
    "window": dict(layers=[(dm.attention(heads=4, kv_heads=2, dim=64, vdim=48, window=48), None)]),
    "window odd": dict(layers=[(dm.attention(heads=3, kv_heads=1, dim=33, vdim=17, window=29), None)]),
    "chunks": dict(layers=[(dm.chunked(heads=4, kv_heads=1, dim=128, vdim=128, rot=64, chunk=90), None)]),
    "chunks odd": dict(layers=[(dm.chunked(heads=3, kv_heads=3, dim=30, vdim=40, rot=22, chunk=65), None)]),
    "recurrent unit": dict(layers=[(dm.rglru(width=256, blocks=1, taps=4), None)]),
    "recurrent unit odd": dict(layers=[(dm.rglru(width=34, blocks=2, taps=3), None)]),
    "recurrent unit of large blocks": dict(layers=[(dm.rglru(width=288, blocks=1, taps=4), None)]),
    "experts": dict(layers=[(dm.rglru(width=16, blocks=1), dm.moe(experts=8, top=3, ff=128, groups=4, keep=2))]),
}


def _model(name, dtype, tmp_path):
    cfg = dm.config(**MODELS[name])
    w = dm.weights(cfg, seed=len(name), decisive=dtype == "bfloat16")
    return cfg, w, dm.save(tmp_path / name, cfg, w)


def _check(got, want, dtype, what):
    worst, mean = dm.errors(got, want)
    assert worst < LIMIT[dtype] and mean < MEAN_LIMIT[dtype], (what, worst, mean)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_portions_decode_and_mixed_batches(name, dtype, tmp_path):
    cfg, w, path = _model(name, dtype, tmp_path)
    prompts = {"a": dm.tokens(301, cfg["vocab"], 1), "b": dm.tokens(150, cfg["vocab"], 2),
               "c": dm.tokens(17, cfg["vocab"], 3), "d": dm.tokens(1, cfg["vocab"], 4)}
    want = dm.expected(cfg, w, prompts)
    whole = [[(i, len(t))] for i, t in prompts.items()]
    together = [[(i, len(t)) for i, t in prompts.items()]]
    cut = [[("a", 2), ("b", 65)], [("a", 64), ("d", 1)], [("b", 1)], [("a", 130), ("b", 1), ("c", 2)],
           [("c", 1), ("b", 1)], [("b", 63), ("a", 1), ("c", 1)], [("a", 60), ("b", 2), ("c", 13)]] + \
          [[("a", 1), ("b", 1)]] * 17 + [[("a", 1)]] * 27
    llm = dm.engine(path, "cuda", dtype)
    for schedule in (whole, together, cut):
        got = dm.feed(llm, prompts, schedule)
        for i in prompts:
            _check(got[i], want[i], dtype, (i, schedule[0]))
    llm.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_in_portions_of_several_sizes(name, dtype, tmp_path):
    cfg = dm.config(**dict(SINGLE[name], width=96, vocab=90))
    w = dm.weights(cfg, seed=11, decisive=dtype == "bfloat16")
    llm = dm.engine(dm.save(tmp_path / "m", cfg, w), "cuda", dtype)
    prompts = {"a": dm.tokens(206, cfg["vocab"], 5)}
    want = dm.expected(cfg, w, prompts)["a"]
    for sizes in ([206], [2] * 103, [64, 64, 64, 14], [63, 1, 65, 1, 76], [30, 1, 25, 150], [130] + [1] * 76):
        got = dm.feed(llm, prompts, [[("a", n)] for n in sizes])["a"]
        _check(got, want, dtype, sizes[:5])
    llm.exit()


def _pointer(spec, at, n, dtype, tmp_path):
    cfg, w, prompt = dm.pointer_model(spec, at, n)
    want = oracle.forward(cfg, w, prompt)[0]
    llm = dm.engine(dm.save(tmp_path / f"m{at}", cfg, w), "cuda", dtype, page=64 if at % 2 else 16, enforce_eager=True)
    for cut in ([n], [n - 1, 1], [at + 1, (n - at - 1) // 2, (n - at) // 2], [256, 129, n - 385], [100, n - 140, 40]):
        got = dm.feed(llm, {"a": prompt}, [[("a", c)] for c in cut if c])["a"]
        worst, _ = dm.errors(got[-1:], want[-1:])
        assert worst < (0.05 if dtype == "bfloat16" else 2e-4), (at, cut, worst)
    llm.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [63, 64, 128, 129, 300])
def test_keys_at_the_edges_of_the_window(window, dtype, tmp_path):
    """One key carries the whole answer, just inside and just outside the window: prompts, portions and decoding."""
    n = 420
    for at in (n - 1 - window, n - window, n - 2):
        _pointer(dm.attention(heads=4, kv_heads=2, dim=64, vdim=64, window=window), at, n, dtype, tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [64, 127, 128, 200, 383, 419])
def test_keys_at_the_edges_of_the_chunk(chunk, dtype, tmp_path):
    n = 420
    first = (n - 1) // chunk * chunk
    for at in sorted({first - 1, min(first, n - 2)} - {-1}):
        _pointer(dm.chunked(heads=4, kv_heads=2, dim=64, vdim=64, rot=32, chunk=chunk, softcap=40.0), at, n, dtype, tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_with_old_contents(dtype, tmp_path):
    cfg, w, path = _model("wide", dtype, tmp_path)
    llm = dm.engine(path, "cuda", dtype, max_tokens=20 * dm.PAGE, requests=2)
    fill_caches(llm, 1e3)
    for k in range(4):
        prompts = {f"x{k}": dm.tokens(130 + k, cfg["vocab"], k), f"y{k}": dm.tokens(90 - 20 * k, cfg["vocab"], 50 + k)}
        want = dm.expected(cfg, w, prompts)
        a, b = prompts
        n, m = len(prompts[a]), len(prompts[b])
        got = dm.feed(llm, prompts, [[(b, 1)], [(a, 100), (b, 3)], [(a, n - 103), (b, 1)], [(b, m - 8), (a, 1)],
                                     [(a, 1), (b, 1)], [(a, 1), (b, 1)], [(b, 1)]])
        for i in prompts:
            _check(got[i], want[i], dtype, i)
    llm.exit()


@pytest.mark.parametrize("name", ["wide", "mid"])
def test_general_kernels_in_bf16(name, tmp_path, monkeypatch):
    from fastcache_b200.ops import hybrid
    monkeypatch.setattr(hybrid, "ATTN_IMPL", 1)
    monkeypatch.setattr(hybrid, "LRU_IMPL", 1)
    cfg, w, path = _model(name, "bfloat16", tmp_path)
    prompts = {"a": dm.tokens(190, cfg["vocab"], 1)}
    llm = dm.engine(path, "cuda", "bfloat16", enforce_eager=True)
    _check(dm.feed(llm, prompts, [[("a", 170)], [("a", 18)], [("a", 1)], [("a", 1)]])["a"],
           dm.expected(cfg, w, prompts)["a"], "bfloat16", "general")
    llm.exit()


def test_long_context_decode_with_splits_and_large_prompts(tmp_path):
    cfg, w, path = _model("mid", "bfloat16", tmp_path)
    n = 1500
    prompts = {"a": dm.tokens(n, cfg["vocab"], 1), "b": dm.tokens(n // 3, cfg["vocab"], 2)}
    want = dm.expected(cfg, w, prompts)
    llm = dm.engine(path, "cuda", "bfloat16", max_tokens=4096)
    got = dm.feed(llm, prompts, [[("a", n - 40), ("b", n // 3 - 40)]] + [[("a", 1), ("b", 1)]] * 40)
    for i in prompts:
        _check(got[i], want[i], "bfloat16", i)
    llm.exit()


@pytest.mark.parametrize("name", ["general", "wide"])
def test_generation_matches_between_graph_and_eager_and_split_prompts(name, tmp_path):
    from fastcache_b200 import SamplingParams
    cfg, w, path = _model(name, "float32", tmp_path)
    prompts = [dm.tokens(n, cfg["vocab"], n) for n in (70, 3, 33, 129, 1)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    outs = []
    for kw in (dict(enforce_eager=True), dict(), dict(max_num_batched_tokens=40, chunked_prefill_tokens=8)):
        llm = dm.engine(path, "cuda", "float32", **kw)
        outs.append([o["token_ids"] for o in llm.generate(prompts, sp)])
        llm.exit()
    assert outs[0] == outs[1] == outs[2]
    seq = prompts[0] + outs[0][0]
    logits = oracle.forward(cfg, w, seq)[0]
    assert logits[len(prompts[0]) - 1:-1].argmax(-1).tolist() == outs[0][0]


# ------------------------------------------------------------------ single ops
def _rnd(*shape, scale=1.0, dtype=torch.bfloat16, seed=0):
    g = torch.Generator(device="cuda").manual_seed(seed)
    return (torch.randn(*shape, device="cuda", generator=g) * scale).to(dtype)


@pytest.mark.parametrize("H,G,D,V,page,window,chunk,cap,sharp",
                         [(8, 2, 128, 128, 64, 0, 400, 30.0, 1.0), (8, 2, 128, 128, 64, 0, 400, 30.0, 6.0), (4, 4, 64, 64, 16, 0, 64, 5.0, 1.0),
                          (16, 1, 96, 64, 256, 1000, 0, 0.0, 1.0), (6, 3, 40, 56, 8, 0, 33, 50.0, 1.0), (2, 1, 128, 72, 32, 0, 0, 20.0, 2.0),
                          (4, 2, 64, 64, 64, 90, 256, 10.0, 1.0), (4, 1, 128, 128, 64, 0, 1100, 0.0, 1.0)])
def test_projected_attention_op(H, G, D, V, page, window, chunk, cap, sharp):
    """Prefill of several requests (whole, continued, short) and decoding with context splits; soft caps that the scores stay
    below, and reach."""
    from fastcache_b200.layers.windowed_attention import padded_dim
    from fastcache_b200.ops import hybrid
    from fastcache_b200.ops.loader import ext
    rot, eps, scale = D // 2, 1e-5, sharp * D ** -0.5
    scaling = dict(factor=4.0, original=256, fast=20.0, slow=1.0)
    ctx = [700, 64, 130, 1, 1290]
    new = {True: [700, 2, 70, 1, 300], False: [1] * 5}
    P = padded_dim(max(D, V))
    pages = -(-max(ctx) // page)
    bt = torch.randperm(5 * pages, generator=torch.Generator().manual_seed(1)).int().view(5, pages)
    N = (H + G) * D + G * V
    hist = [_rnd(n, N, seed=i) for i, n in enumerate(ctx)]
    bias = _rnd(N, scale=0.5, seed=20)
    q_norm, k_norm = _rnd(H * D, dtype=torch.float32, seed=7).abs() + 1.5, _rnd(G * D, dtype=torch.float32, seed=8).abs() + 0.5
    freq = hybrid.rope_turns(1e4, rot, scaling).cuda()
    d = hybrid.WindowDims(H, G, D, rot, scale, window, 0, H * D, None, (H + G) * D, V, chunk, cap, True, hybrid.rope_size(scaling))
    for prefill in (True, False):
        pools = [torch.full((5 * pages, G, page, P), 50.0, device="cuda", dtype=torch.bfloat16) for _ in range(2)]

        def run(lens, start, is_prefill):
            rows = torch.cat([hist[i][s:s + n] for i, (s, n) in enumerate(zip(start, lens))])
            pos = torch.cat([torch.arange(s, s + n) for s, n in zip(start, lens)]).cuda()
            seq = torch.repeat_interleave(torch.arange(5), torch.tensor(lens))
            slots = (bt[seq, pos.cpu() // page] * page + pos.cpu() % page).int().cuda()
            out = torch.full((rows.shape[0], -(-H * V // 8) * 8), 7.0, device="cuda", dtype=torch.bfloat16)
            end = torch.tensor([s + n for s, n in zip(start, lens)], dtype=torch.int32, device="cuda")
            cu = torch.tensor([0] + lens, dtype=torch.int32).cumsum(0).int().cuda() if is_prefill else None
            ext().windowed_attention(ext().as_projection(rows), d.sizes(), d.scale, d.softcap, d.rot_size, freq, bias, q_norm, k_norm,
                                     None, eps, *pools, pos, slots, bt.cuda(), end, cu, seq.int().cuda() if is_prefill else None,
                                     (pos + 1).int() if is_prefill else None, max(lens), 0, out, 0)
            return out

        lens = new[prefill]
        start = [n - k for n, k in zip(ctx, lens)]
        if any(start):
            run([max(s, 1) for s in start], [0] * 5, True)
        got = run(lens, start, prefill).float().cpu()
        at = 0
        for i, (s, k) in enumerate(zip(start, lens)):
            x = (hist[i].float() + bias.float()).cpu().double()
            n, p = ctx[i], torch.arange(ctx[i])
            r = dict(base=1e4, dims=rot, scaling=scaling)
            q = oracle.rotate_half((oracle.rms(x[:, :H * D], eps) * q_norm.cpu().double()).view(n, H, D), p, r)
            kn = oracle.rotate_half((oracle.rms(x[:, H * D:(H + G) * D], eps) * k_norm.cpu().double()).view(n, G, D), p, r)
            # what the pages and the queries hold: 16-bit rows
            q, kn = (t.bfloat16().double() for t in (q, kn))
            v = x[:, (H + G) * D:].reshape(n, G, V)
            kn, v = (t.repeat_interleave(H // G, 1) for t in (kn, v))
            sc = torch.einsum("ihd,jhd->hij", q[s:], kn) * scale
            if cap:
                sc = cap * torch.tanh(sc / cap)
            a, b = p[s:, None], p[None]
            seen = oracle.chunks(a, b, chunk or n)
            if window:
                seen &= oracle.sliding_window(a, b, window)
            want = torch.einsum("hij,jhd->ihd", torch.softmax(sc.masked_fill(~seen, float("-inf")), -1), v).reshape(k, H * V)
            assert (got[at:at + k, :H * V] - want).abs().max() < 0.06, (prefill, i)
            assert (got[at:at + k, H * V:] == 0).all()
            at += k
    assert ext().read_status(0) == 0


@pytest.mark.parametrize("E,groups,keep,top", [(6, 3, 2, 2), (8, 1, 1, 8), (16, 4, 1, 4), (12, 12, 5, 3), (64, 8, 4, 6), (160, 5, 2, 33),
                                               (256, 8, 3, 8), (1, 1, 1, 1)])
@pytest.mark.parametrize("T,dtype", [(1, torch.bfloat16), (37, torch.float32), (256, torch.bfloat16), (700, torch.bfloat16)])
def test_route_by_score_op(E, groups, keep, top, T, dtype):
    from fastcache_b200.layers.linear import pad8
    from fastcache_b200.ops import hybrid
    from fastcache_b200.utils.context import Context
    K = 64
    h = _rnd(T, K, dtype=dtype, seed=T)
    w = torch.zeros(pad8(E), K, device="cuda", dtype=dtype)
    w[:E] = _rnd(E, K, scale=2 * K ** -0.5, dtype=dtype, seed=E)
    c = _rnd(E, scale=0.4, dtype=torch.float32, seed=3) - 0.6
    decode = T <= 256
    ctx = Context(is_prefill=not decode, context_lens=(torch.arange(T, device="cuda") % 5 != 3).int())
    (row_of, plan), mix = hybrid.route_by_score(h, w, c, top, groups, keep, ctx)
    row_of, plan, mix = row_of.cpu(), plan.cpu(), mix.cpu()
    z = (h.double() @ w[:E].double().T).cpu()
    router = dict(experts=E, top=top, groups=dict(count=groups, keep=keep))
    first = plan[:E + 1].tolist()
    used = 0
    for t in range(T):
        rows = row_of[t].tolist()
        if decode and t % 5 == 3:
            assert rows == [-1] * top
            continue
        want = oracle.route(z[t], c.cpu().double(), router)
        ids = [next(e for e in range(E) if first[e] <= r < first[e + 1]) for r in rows]
        assert sorted(ids) == sorted(want), t
        assert all(abs(float(mix[t, j]) - float(want[e])) < 1e-4 for j, e in enumerate(ids)), t
        used += top
    assert first[0] == 0 and first[E] == used
    tiles = int(plan[E + 1])
    pairs = [(int(plan[E + 2 + 2 * i]), int(plan[E + 3 + 2 * i])) for i in range(tiles)]
    assert pairs == [(e, r) for e in range(E) for r in range(first[e], first[e + 1], 128)]
    token = plan[-T * top:]
    assert all(int(token[r]) == t for t in range(T) for r in row_of[t].tolist() if r >= 0)


@pytest.mark.parametrize("S", [1, 2, 3, 4, 6, 11])
@pytest.mark.parametrize("T,W", [(3, 72), (3, 61), (400, 1500), (200, 4096), (310, 6000), (5, 8192)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_streams_op(S, T, W, dtype):
    from fastcache_b200.layers.linear import pad8
    from fastcache_b200.ops import hybrid
    eps = 1e-5
    x, y = _rnd(T, S, W, dtype=torch.float32), torch.zeros(T, pad8(W), device="cuda", dtype=dtype)
    y[:, :W] = _rnd(T, W, dtype=dtype, seed=1)
    hc, nxt = (_rnd(S * (S + 2), dtype=torch.float32, seed=2 + k) for k in range(2))
    w, b = _rnd(W, dtype=torch.float32, seed=5), _rnd(W, dtype=torch.float32, seed=6)

    def parts(c):
        c = c.double().cpu()
        return {"in": c[:S], "out": c[S:2 * S], "mix": c[2 * S:].view(S, S)}

    from fastcache_b200.ops.loader import ext
    new = oracle.streams_out(x.double().cpu(), y[:, :W].double().cpu(), parts(hc))
    for c in (nxt, None):
        z = x.clone()
        h = ext().mix_norm(ext().as_projection(y), z, hc, c, w, b, eps)
        u = new.sum(1) if c is None else oracle.streams_in(new, parts(c))
        want = oracle.layer_norm(u, w.double().cpu(), b.double().cpu(), eps)
        assert (z.cpu() - (x.cpu() if c is None else new)).abs().max() < 1e-4
        assert (h[:, :W].cpu() - want).abs().max() < (0.05 if dtype == torch.bfloat16 else 1e-4)
        assert (h[:, W:] == 0).all()
    table = torch.zeros(9, pad8(W), device="cuda", dtype=dtype)
    table[:, :W] = _rnd(9, W, dtype=dtype, seed=8)
    ids = torch.arange(T, device="cuda") % 9
    z, h = hybrid.embed_streams(ids, table, W, S, (nxt, w, b), eps)
    e = table[ids, :W].double().cpu()[:, None].repeat(1, S, 1)
    assert torch.equal(z.cpu().double(), e)
    want = oracle.layer_norm(oracle.streams_in(e, parts(nxt)), w.double().cpu(), b.double().cpu(), eps)
    assert (h[:, :W].cpu() - want).abs().max() < (0.05 if dtype == torch.bfloat16 else 1e-4)


@pytest.mark.parametrize("C,blocks,taps", [(256, 1, 4), (512, 4, 4), (160, 2, 3), (384, 2, 2), (48, 3, 4), (64, 4, 1), (320, 4, 6)])
def test_recurrent_unit_on_tensor_cores_against_the_plain_one(C, blocks, taps):
    """Outputs and states of long runs (also cut into segments), continued, and single steps; decays from none to full."""
    from fastcache_b200.ops.loader import ext
    n, W = C // blocks, 64
    lens = [1, 200, 64, 2333]
    T = sum(lens)
    h, wt = _rnd(T, W), _rnd(2 * C, W, scale=W ** -0.5, seed=1)
    bias = _rnd(2 * C, scale=0.3, seed=2)
    cw, cb = _rnd(C, taps, scale=0.6, dtype=torch.float32, seed=3), _rnd(C, scale=0.3, dtype=torch.float32, seed=4)
    gw, gb = _rnd(2, blocks, n, n, scale=2 * n ** -0.5, seed=5), _rnd(2, C, scale=0.5, dtype=torch.float32, seed=6)
    lam = torch.linspace(-9, 3, C, device="cuda")
    slots = torch.tensor([3, 0, 2, 1], dtype=torch.int32, device="cuda")
    base = [sum(lens[:i]) for i in range(4)]
    outs, states = {}, {}
    for impl in (0, 1):
        st, cs = torch.full((4, C), 9.0, device="cuda"), torch.full((4, taps - 1, C), 9.0, device="cuda")
        got = [[] for _ in lens]

        def run(parts):
            """parts: (first, count) per request; one row each is a decode step"""
            cut = [c for _, c in parts]
            idx = torch.cat([torch.arange(b + f, b + f + c) for b, (f, c) in zip(base, parts)]).cuda()
            ctx = torch.tensor([f + c for f, c in parts], dtype=torch.int32, device="cuda")
            prefill = any(c != 1 for c in cut) or any(f == 0 for f, _ in parts)
            cu = torch.tensor([0] + cut, dtype=torch.int32).cumsum(0).int().cuda() if prefill else None
            seq = torch.repeat_interleave(torch.arange(4), torch.tensor(cut)).int().cuda() if prefill else None
            o = ext().real_gated_lru(h[idx].contiguous(), wt, bias, [C, blocks, 0, C], 8.0, cw, cb, gw, gb, lam, cs, st, cu, ctx, slots,
                                     max(cut), seq, impl).float()
            for i, piece in enumerate(o[:, :C].split(cut)):
                got[i].append(piece.cpu())

        run([(0, 1), (0, 70), (0, 2), (0, 2100)])
        run([(0, 1), (70, 1), (2, 1), (2100, 231)])
        for k in range(2):
            run([(0, 1), (71 + k, 1), (3 + k, 1), (2331 + k, 1)] if k == 0 else [(0, 1), (72, 1), (4, 1), (2332, 1)])
        run([(0, 1), (73, 127), (5, 59), (2332, 1)])
        outs[impl] = [torch.cat([g[0] for g in [x]] if i == 0 else x) for i, x in enumerate(got)]
        states[impl] = (st.cpu(), cs.cpu())
    hd, wd, bd = h.double().cpu(), wt.double().cpu(), bias.double().cpu()
    for i in (1, 2):
        x = hd[base[i]:base[i] + lens[i]]
        y = oracle.gelu_tanh(x @ wd[:C].T + bd[:C])
        u = oracle.causal_conv(x @ wd[C:].T + bd[C:], cw.double().cpu(), cb.double().cpu())
        r, g = (oracle.sigmoid(oracle.block_linear(u, gw[m].double().cpu(), gb[m].view(blocks, n).double().cpu())) for m in (0, 1))
        s = oracle.lru_scan(u, r, g, lam.double().cpu())
        for impl in (0, 1):
            got = outs[impl][i][:lens[i]]
            assert (got - s * y).abs().max() < 0.05 * max(1.0, float((s * y).abs().max())), (impl, i)
            assert (states[impl][0][slots[i]] - s[-1]).abs().max() < 0.03 * max(1.0, float(s.abs().max())), (impl, i)
    for a, b in zip(outs[0], outs[1]):
        assert (a - b).abs().max() < 0.03 * max(1.0, float(b.abs().max()))
    assert ext().read_status(0) == 0
