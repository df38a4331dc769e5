"""Lekilix on a CUDA device: the engine's kernels in bf16 and fp32 against the plain implementation."""
import math

import pytest
import torch

import lekilix_models as lm
import lekilix_oracle as oracle
from test_lekilix_cpu import fill_caches

pytestmark = pytest.mark.gpu

LIMIT = {"bfloat16": 0.2, "float32": 2e-4}            # worst position
MEAN_LIMIT = {"bfloat16": 0.03, "float32": 2e-5}      # all positions

# sizes for the tensor-core forms and sizes that only the general kernels take
MODELS = {
    "general": dict(layers=[(lm.mlstm(), lm.dense()), (lm.attention(), lm.moe()), (lm.mlstm(heads=2, dim=16, vdim=48), lm.moe()),
                            (lm.attention(window=70), None)], loop=(1, 3, 2)),
    "odd": dict(layers=[(lm.attention(heads=5, kv_heads=1, dim=13, rot=6, window=37), lm.moe(experts=3, top=1, ff=11)),
                        (lm.mlstm(heads=1, dim=7, vdim=9), lm.dense(45)), (lm.mlstm(heads=3, dim=5, vdim=130), None),
                        (lm.attention(heads=2, kv_heads=2, dim=150, rot=150, window=64), None)], width=61, vocab=77, loop=(0, 2, 2)),
    "wide": dict(layers=[(lm.attention(heads=4, kv_heads=2, dim=128, rot=64, window=100), lm.dense(384)),
                         (lm.mlstm(heads=2, dim=128, vdim=128), lm.moe(experts=8, top=2, ff=128)),
                         (lm.attention(heads=8, kv_heads=1, dim=64, rot=64, window=128), lm.moe(experts=4, top=2, ff=256)),
                         (lm.mlstm(heads=2, dim=64, vdim=256), lm.dense(256))], width=256, vocab=520, loop=(2, 4, 2)),
    "mid": dict(layers=[(lm.attention(heads=6, kv_heads=3, dim=96, rot=32, window=300), lm.dense(96)),
                        (lm.mlstm(heads=4, dim=32, vdim=64), lm.moe(experts=16, top=4, ff=64))], width=128, vocab=200),
    "many heads": dict(layers=[(lm.attention(heads=36, kv_heads=2, dim=32, rot=8, window=90), None),
                               (lm.mlstm(heads=12, dim=16, vdim=16), lm.dense(128))], width=192, vocab=100, loop=(0, 1, 3)),
}
SINGLE = {
    "attention": dict(layers=[(lm.attention(heads=4, kv_heads=2, dim=64, rot=32, window=48), None)]),
    "attention odd": dict(layers=[(lm.attention(heads=3, kv_heads=1, dim=33, rot=10, window=29), None)]),
    "mlstm": dict(layers=[(lm.mlstm(heads=2, dim=48, vdim=80, cap=12.0), None)]),
    "mlstm odd": dict(layers=[(lm.mlstm(heads=2, dim=33, vdim=35), None)]),
    "mlstm several column blocks": dict(layers=[(lm.mlstm(heads=2, dim=20, vdim=270), None)]),
    "experts": dict(layers=[(lm.mlstm(heads=1, dim=8, vdim=8), lm.moe(experts=7, top=3, ff=128))]),
}


def _model(name, tmp_path):
    cfg = lm.config(**MODELS[name])
    w = lm.weights(cfg, seed=len(name))
    return cfg, w, lm.save(tmp_path / name, cfg, w)


def _check(got, want, dtype, what):
    """Every position in 32-bit; in bf16 all but one in a hundred: where n.q of a matrix memory crosses zero its normalised
    output turns around, and rounding alone decides how far."""
    if dtype == "bfloat16":
        each = torch.tensor([lm.errors(got[i:i + 1], want[i:i + 1])[0] for i in range(len(got))]).sort().values
        worst, mean = float(each[len(each) - 1 - max(1, len(each) // 100)]) if len(each) > 2 else float(each[0]), float(each.mean())
    else:
        worst, mean = lm.errors(got, want)
    assert worst < LIMIT[dtype] and mean < MEAN_LIMIT[dtype], (what, worst, mean)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_portions_decode_and_mixed_batches(name, dtype, tmp_path):
    cfg, w, path = _model(name, tmp_path)
    prompts = {"a": lm.tokens(301, cfg["vocab"], 1), "b": lm.tokens(150, cfg["vocab"], 2),
               "c": lm.tokens(17, cfg["vocab"], 3), "d": lm.tokens(1, cfg["vocab"], 4)}
    want = lm.expected(cfg, w, prompts)
    whole = [[(i, len(t))] for i, t in prompts.items()]
    together = [[(i, len(t)) for i, t in prompts.items()]]
    cut = [[("a", 2), ("b", 65)], [("a", 64), ("d", 1)], [("b", 1)], [("a", 130), ("b", 1), ("c", 2)],
           [("c", 1), ("b", 1)], [("b", 63), ("a", 1), ("c", 1)], [("a", 60), ("b", 2), ("c", 13)]] + \
          [[("a", 1), ("b", 1)]] * 17 + [[("a", 1)]] * 27
    llm = lm.engine(path, "cuda", dtype)
    for schedule in (whole, together, cut):
        got = lm.feed(llm, prompts, schedule)
        for i in prompts:
            _check(got[i], want[i], dtype, (i, schedule[0]))
    llm.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_in_portions_of_several_sizes(name, dtype, tmp_path):
    cfg = lm.config(**dict(SINGLE[name], width=96, vocab=90))
    w = lm.weights(cfg, seed=11)
    llm = lm.engine(lm.save(tmp_path / "m", cfg, w), "cuda", dtype)
    prompts = {"a": lm.tokens(206, cfg["vocab"], 5)}
    want = lm.expected(cfg, w, prompts)["a"]
    for sizes in ([206], [2] * 103, [64, 64, 64, 14], [63, 1, 65, 1, 76], [30, 1, 25, 150], [130] + [1] * 76):
        got = lm.feed(llm, prompts, [[("a", n)] for n in sizes])["a"]
        _check(got, want, dtype, sizes[:5])
    llm.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [63, 64, 127, 128, 129, 256, 300])
def test_keys_at_the_edges_of_the_window(window, dtype, tmp_path):
    """One key carries the whole answer, just inside and just outside the window: prompts, portions and decoding."""
    n = 420
    for at in (n - 1 - window, n - window, n - 2):
        cfg, w, prompt = lm.pointer_model(lm.attention(heads=4, kv_heads=2, dim=64, rot=32, window=window), at, n)
        want = oracle.forward(cfg, w, prompt)[0]
        llm = lm.engine(lm.save(tmp_path / f"m{at}", cfg, w), "cuda", dtype, page=64 if at % 2 else 16, enforce_eager=True)
        for cut in ([n], [n - 1, 1], [at + 1, n - at - 3, 2], [256, 129, n - 385], [100, n - 140, 40]):
            got = lm.feed(llm, {"a": prompt}, [[("a", c)] for c in cut if c])["a"]
            worst, _ = lm.errors(got[-1:], want[-1:])
            assert worst < (0.05 if dtype == "bfloat16" else 2e-4), (at, cut, worst)
        llm.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_with_old_contents(dtype, tmp_path):
    cfg, w, path = _model("wide", tmp_path)
    llm = lm.engine(path, "cuda", dtype, max_tokens=20 * lm.PAGE, requests=2)
    fill_caches(llm, 1e3)
    for k in range(4):
        prompts = {f"x{k}": lm.tokens(130 + k, cfg["vocab"], k), f"y{k}": lm.tokens(90 - 20 * k, cfg["vocab"], 50 + k)}
        want = lm.expected(cfg, w, prompts)
        a, b = prompts
        n, m = len(prompts[a]), len(prompts[b])
        got = lm.feed(llm, prompts, [[(b, 1)], [(a, 100), (b, 3)], [(a, n - 103), (b, 1)], [(b, m - 8), (a, 1)],
                                     [(a, 1), (b, 1)], [(a, 1), (b, 1)], [(b, 1)]])
        for i in prompts:
            _check(got[i], want[i], dtype, i)
    llm.exit()


@pytest.mark.parametrize("name", ["wide", "mid"])
def test_general_attention_kernel_in_bf16(name, tmp_path, monkeypatch):
    from fastcache_b200.ops import hybrid
    monkeypatch.setattr(hybrid, "ATTN_IMPL", 1)
    cfg, w, path = _model(name, tmp_path)
    prompts = {"a": lm.tokens(190, cfg["vocab"], 1)}
    llm = lm.engine(path, "cuda", "bfloat16", enforce_eager=True)
    _check(lm.feed(llm, prompts, [[("a", 170)], [("a", 18)], [("a", 1)], [("a", 1)]])["a"],
           lm.expected(cfg, w, prompts)["a"], "bfloat16", "general")
    llm.exit()


def test_long_context_decode_with_splits_and_large_prompts(tmp_path):
    cfg, w, path = _model("mid", tmp_path)
    n = 1500
    prompts = {"a": lm.tokens(n, cfg["vocab"], 1), "b": lm.tokens(n // 3, cfg["vocab"], 2)}
    want = lm.expected(cfg, w, prompts)
    llm = lm.engine(path, "cuda", "bfloat16", max_tokens=4096)
    got = lm.feed(llm, prompts, [[("a", n - 40), ("b", n // 3 - 40)]] + [[("a", 1), ("b", 1)]] * 40)
    for i in prompts:
        _check(got[i], want[i], "bfloat16", i)
    llm.exit()


@pytest.mark.parametrize("name", ["general", "wide"])
def test_generation_matches_between_graph_and_eager_and_split_prompts(name, tmp_path):
    from fastcache_b200 import SamplingParams
    cfg, w, path = _model(name, tmp_path)
    prompts = [lm.tokens(n, cfg["vocab"], n) for n in (70, 3, 33, 129, 1)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    outs = []
    for kw in (dict(enforce_eager=True), dict(), dict(max_num_batched_tokens=40, chunked_prefill_tokens=8)):
        llm = lm.engine(path, "cuda", "float32", **kw)
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


@pytest.mark.parametrize("H,G,D,page,window", [(8, 2, 128, 64, 200), (4, 4, 64, 16, 64), (16, 1, 96, 256, 1000), (6, 3, 40, 8, 33),
                                               (2, 1, 128, 32, 0)])
def test_windowed_attention_op(H, G, D, page, window):
    """Prefill of several requests (whole, continued, short) and decoding with context splits, peaked scores, strong sinks."""
    from fastcache_b200.layers.windowed_attention import padded_dim
    from fastcache_b200.ops.hybrid import WindowDims, rope_turns
    from fastcache_b200.ops.loader import ext
    rot, eps, base, scale = D // 2, 1e-5, 1e4, D ** -0.5
    ctx = [700, 64, 130, 1, 1290]
    new = {True: [700, 2, 70, 1, 300], False: [1] * 5}
    P = padded_dim(D)
    pages = -(-max(ctx) // page)
    bt = torch.randperm(5 * pages, generator=torch.Generator().manual_seed(1)).int().view(5, pages)
    hist = [_rnd(n, (2 * H + G) * D, seed=i) for i, n in enumerate(ctx)]
    q_norm, k_norm = _rnd(H * D, dtype=torch.float32, seed=7).abs() + 1.5, _rnd(G * D, dtype=torch.float32, seed=8).abs() + 0.5
    sink = _rnd(H, scale=3.0, dtype=torch.float32, seed=9)
    freq = rope_turns(base, rot).cuda()
    cols = WindowDims(H, G, D, rot, scale, window, 0, H * D, (H + G) * D).sizes()
    for prefill in (True, False):
        pools = [torch.full((5 * pages, G, page, P), 50.0, device="cuda", dtype=torch.bfloat16) for _ in range(2)]

        def run(lens, start, is_prefill):
            rows = torch.cat([hist[i][s:s + n] for i, (s, n) in enumerate(zip(start, lens))])
            pos = torch.cat([torch.arange(s, s + n) for s, n in zip(start, lens)]).cuda()
            seq = torch.repeat_interleave(torch.arange(5), torch.tensor(lens))
            slots = (bt[seq, pos.cpu() // page] * page + pos.cpu() % page).int().cuda()
            out = torch.full((rows.shape[0], -(-H * D // 8) * 8), 7.0, device="cuda", dtype=torch.bfloat16)
            end = torch.tensor([s + n for s, n in zip(start, lens)], dtype=torch.int32, device="cuda")
            cu = torch.tensor([0] + lens, dtype=torch.int32).cumsum(0).int().cuda() if is_prefill else None
            ext().windowed_attention(ext().as_projection(rows), cols, scale, 0.0, 1.0, freq, None, q_norm, k_norm, sink, eps, *pools, pos, slots,
                                     bt.cuda(), end, cu, seq.int().cuda() if is_prefill else None,
                                     (pos + 1).int() if is_prefill else None, max(lens), 0, out, 0)
            return out

        lens = new[prefill]
        start = [n - k for n, k in zip(ctx, lens)]
        if any(start):
            run([max(s, 1) for s in start], [0] * 5, True)
        got = run(lens, start, prefill).float().cpu()
        at = 0
        for i, (s, k) in enumerate(zip(start, lens)):
            x = hist[i].cpu().double()
            n, p = ctx[i], torch.arange(ctx[i])
            q = oracle.rotate_pairs((oracle.rms(x[:, :H * D], eps) * q_norm.cpu().double()).view(n, H, D), p, rot, base)
            kk = x[:, H * D:(H + G) * D]
            kn = oracle.rotate_pairs((oracle.rms(kk, eps) * k_norm.cpu().double()).view(n, G, D), p, rot, base)
            kn, v = (t.reshape(n, G, D).repeat_interleave(H // G, 1) for t in (kn, kk))
            sc = torch.einsum("ihd,jhd->hij", q[s:], kn) * scale
            back = p[s:, None] - p[None]
            sc = sc.masked_fill((back < 0) | (back >= (window or n)), float("-inf"))
            o = torch.einsum("hij,jhd->ihd", oracle.sink_softmax(sc, sink.cpu().double()), v).reshape(k, H * D)
            want = o * torch.sigmoid(x[s:, (H + G) * D:])
            assert (got[at:at + k, :H * D] - want).abs().max() < 0.06, (prefill, i)
            assert (got[at:at + k, H * D:] == 0).all()
            at += k
    assert ext().read_status(0) == 0


@pytest.mark.parametrize("T,W,E,top,ff,dtype", [(300, 192, 8, 2, 128, torch.bfloat16), (1000, 320, 5, 3, 40, torch.bfloat16),
                                                (64, 512, 16, 4, 256, torch.bfloat16), (1, 264, 7, 2, 136, torch.bfloat16),
                                                (200, 128, 3, 1, 64, torch.bfloat16), (130, 72, 4, 2, 24, torch.float32)])
@pytest.mark.parametrize("act", ["clamped", "silu"])
def test_experts_op(T, W, E, top, ff, dtype, act):
    from fastcache_b200.layers.linear import pad8
    from fastcache_b200.ops import hybrid
    from fastcache_b200.utils.context import Context
    vocab, fp = 50, pad8(ff)
    g = torch.Generator().manual_seed(T)
    table = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(vocab)]).int().cuda()
    if T == 1000:
        table[:] = torch.tensor([0, 2, 4])                   # experts without rows beside full ones
    ids = torch.randint(0, vocab, (T,), generator=g).cuda()
    h = _rnd(T, W, dtype=dtype)
    gu = torch.zeros(E, 2 * fp, W, device="cuda", dtype=dtype)
    gu[:, :ff], gu[:, fp:fp + ff] = _rnd(E, ff, W, scale=2 * W ** -0.5, dtype=dtype, seed=1), _rnd(E, ff, W, scale=2 * W ** -0.5, dtype=dtype, seed=2)
    down = torch.zeros(E, W, fp, device="cuda", dtype=dtype)
    down[:, :, :ff] = _rnd(E, W, ff, scale=ff ** -0.5, dtype=dtype, seed=3)
    spec = hybrid.GluSpec(act, 1.5)
    mix = torch.rand(T, top, device="cuda") if E == 8 else None
    # decode: every fourth row is padding
    ctx = Context(is_prefill=T > 256, context_lens=(torch.arange(T, device="cuda") % 4 != 3).int())
    route = hybrid.route_by_table(ids, table, E, ctx)
    y = hybrid.experts(h, route, mix, gu, down, ff, spec)
    x = torch.zeros(T, W, device="cuda")
    zero = torch.zeros(W, 8, device="cuda", dtype=dtype)
    got = hybrid.linear_add_norm(torch.zeros(T, 8, device="cuda", dtype=dtype), zero, x, None, 1e-6, experts=y)
    from fastcache_b200.ops import reference_hybrid as ref
    want = ref.experts(h.double().cpu().float(), table[ids].long().cpu(), None if mix is None else mix.cpu(), gu.float().cpu(),
                       down.float().cpu(), ff, act, 1.5)
    if T <= 256:
        want[3::4] = 0
    tol = 2e-4 if dtype == torch.float32 else 0.05
    assert (x.cpu() - want).abs().max() < tol * max(1.0, float(want.abs().max()))
    assert torch.equal(got[:, :W].float(), x.to(dtype).float())


@pytest.mark.parametrize("M", [3, 200, 300, 1000])
def test_projection_forms(M):
    """fp32 columns, fp32 accumulation and the fused gates of packed products."""
    from fastcache_b200.ops.loader import ext
    K, N, W = 200, 328, 100
    x, w = _rnd(M, K), _rnd(N, K, scale=K ** -0.5, seed=1)
    want = (x.float() @ w.float().T).cpu()
    p = ext().project(x, w, 304, 256, 40, M == 200)
    out = torch.empty(M, 104, device="cuda", dtype=torch.bfloat16)
    ext().glu(p, 0, 104, 101, 0, 0.0, out)
    ref = torch.nn.functional.silu(want[:, :101]) * want[:, 104:205]
    assert ((out[:, :101].float().cpu() - ref).abs() / (1 + ref.abs())).max() < 0.025 and (out[:, 101:] == 0).all()
    wd = _rnd(104, K, scale=K ** -0.5, seed=2)
    wd[W:] = 0
    acc = _rnd(M, W, dtype=torch.float32, seed=3)
    norm = _rnd(W, dtype=torch.float32, seed=4)
    for add in (True, False):
        y = acc.clone()
        h = ext().linear_add_norm(x, wd, y, norm, 1e-5, add, None, None, None, None)
        ref = (acc.cpu() if add else 0) + (x.float() @ wd.float().T).cpu()[:, :W]
        assert (y.cpu() - ref).abs().max() < 2e-4
        assert (h[:, :W].float().cpu() - oracle.rms(ref, 1e-5) * norm.cpu()).abs().max() < 0.04 and (h[:, W:] == 0).all()
    ff = 128
    wg = _rnd(2 * ff, K, scale=2 * K ** -0.5, seed=5)
    gu = (x.float() @ wg.float().T).cpu()
    for kind, ref in ((0, torch.nn.functional.silu(gu[:, :ff]) * gu[:, ff:]), (1, oracle.clamped_glu(gu[:, :ff], gu[:, ff:], 1.2))):
        out = torch.empty(M, ff, device="cuda", dtype=torch.bfloat16)
        ext().linear_glu(x, wg, ff, ff, kind, 1.2, out)
        assert ((out.float().cpu() - ref).abs() / (1 + ref.abs())).max() < 0.025


@pytest.mark.parametrize("H,D,V", [(4, 64, 64), (3, 128, 128), (2, 32, 48), (2, 16, 200), (1, 126, 34)])
def test_chunked_matrix_memory_against_token_by_token(H, D, V):
    """Outputs and states of long runs, continued in the middle of a chunk, with gates from sharp to flat."""
    from fastcache_b200.ops.loader import ext
    wide = 2 * H
    off = [0, H * D, 2 * H * D, 2 * H * D + H * V, 2 * H * D + 2 * H * V]
    cols = -(-(off[-1] + wide) // 8) * 8
    lens = [1, 200, 64, 331]
    T = sum(lens)
    pr = _rnd(T, cols)
    gates = _rnd(T, wide, scale=4.0, dtype=torch.float32, seed=1)
    ib, fb = _rnd(H, dtype=torch.float32, seed=2), torch.linspace(-2, 6, H, device="cuda")
    nw = _rnd(H * V, dtype=torch.float32, seed=3)
    d = [H, D, V, *off, off[-1] + H]
    states = {}
    outs = {}
    slots = torch.tensor([3, 0, 2, 1], dtype=torch.int32, device="cuda")
    for form in ("float32", "chunks"):
        st = [torch.full((4, H, D, V), 9.0, device="cuda"), torch.full((4, H, D), 9.0, device="cuda"), torch.full((4, H), 9.0, device="cuda")]
        out = []
        for part in (0, 1):
            cut = [n // 3 if part == 0 else n - n // 3 for n in lens]
            begin = [0 if part == 0 else n // 3 for n in lens]
            first = [sum(lens[:i]) + b for i, b in enumerate(begin)]
            idx = torch.cat([torch.arange(f, f + c) for f, c in zip(first, cut)]).cuda()
            cu = torch.tensor([0] + cut, dtype=torch.int32).cumsum(0).int().cuda()
            ctx = torch.tensor([b + c for b, c in zip(begin, cut)], dtype=torch.int32, device="cuda")
            rows, g = pr[idx].contiguous(), gates[idx].contiguous()
            if form == "float32":
                rows = rows.float()
                rows[:, off[-1]:off[-1] + wide] = g
                p = ext().as_projection(rows)
            else:
                p = ext().as_projection(rows, off[-1], g)
            o = torch.empty(len(idx), -(-H * V // 8) * 8, device="cuda", dtype=rows.dtype)
            ext().matrix_memory(p, d, 8.0, 1e-6, ib, fb, nw, 1e-5, *st, cu, ctx, slots, max(cut), o)
            out.append(o.float())
        states[form], outs[form] = st, torch.cat(out)
    q = pr[:, :H * D].double().cpu().view(T, H, D) * D ** -0.5
    k, v = pr[:, off[1]:off[2]].double().cpu().view(T, H, D), pr[:, off[2]:off[3]].double().cpu().view(T, H, V)
    gi = 8 * torch.tanh((gates[:, :H] + ib).double().cpu() / 8)
    gf = -torch.logaddexp(-8 * torch.tanh((gates[:, H:] + fb).double().cpu() / 8), torch.zeros(T, H, dtype=torch.float64))
    a = sum(lens[:3])
    o = oracle.matrix_memory_scan(q[a:], k[a:], v[a:], gi[a:], gf[a:])
    want = oracle.rms(o, 1e-5).reshape(-1, H * V) * nw.double().cpu() * torch.sigmoid(pr[a:, off[3]:off[4]].double().cpu())
    n3 = lens[3] // 3
    got = torch.cat([outs["float32"][sum(n // 3 for n in lens) - n3:sum(n // 3 for n in lens)], outs["float32"][-(lens[3] - n3):]])
    assert (got.cpu()[:, :H * V] - want).abs().max() < 1e-3
    assert (outs["chunks"] - outs["float32"]).abs().max() < 0.05
    for x, y in zip(states["chunks"], states["float32"]):
        assert (x - y).abs().max() < 2e-5 * max(1.0, float(y.abs().max()))
    assert math.isfinite(float(states["chunks"][0].sum()))
