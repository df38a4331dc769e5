"""Darusun on a CUDA device: the engine's kernels in bf16 and fp32 against the plain statements."""
import pytest
import torch

import darusun_models as dm
import darusun_oracle as oracle
from test_darusun_cpu import fill_caches

pytestmark = pytest.mark.gpu

LIMIT = {"bfloat16": 0.15, "float32": 1e-4}           # worst position
MEAN_LIMIT = {"bfloat16": 0.02, "float32": 1e-5}      # all positions

# sizes for the tensor-core forms and sizes that only the general kernels take
MODELS = {
    "general": dict(layers=[(dm.talking(), dm.moe()), (dm.latent(), dm.dense()), (dm.talking(scale=0.2, kv_from=0), None),
                            (dm.latent(window=70), dm.moe(experts=9, top=4, ff=17, shared=50))]),
    "odd": dict(layers=[(dm.talking(heads=5, kv_heads=1, dim=13, vdim=22, rot=6), dm.dense(45)),
                        (dm.latent(heads=3, dim=11, rot=6, vdim=21, rank=37, q_rank=19, window=37), dm.moe(experts=3, top=1, ff=11, shared=13)),
                        (dm.talking(heads=9, kv_heads=3, dim=15, vdim=9, rot=14), None)], width=61, vocab=77),
    "wide": dict(layers=[(dm.talking(heads=8, kv_heads=2, dim=64, vdim=48, rot=48), dm.dense(384)),
                         (dm.latent(heads=4, dim=64, rot=32, vdim=64, rank=192, q_rank=96, window=100), dm.moe(experts=8, top=2, ff=128, shared=256)),
                         (dm.talking(heads=8, kv_heads=2, dim=64, vdim=48, rot=48, scale=0.06, kv_from=0), dm.moe(experts=4, top=2, ff=256, shared=128)),
                         (dm.latent(heads=8, dim=40, rot=24, vdim=56, rank=128, q_rank=64, window=33), None)], width=256, vocab=520),
    "mid": dict(layers=[(dm.talking(heads=6, kv_heads=3, dim=112, vdim=80, rot=64, scale=0.1), dm.dense(96)),
                        (dm.latent(heads=2, dim=120, rot=64, vdim=128, rank=512, q_rank=72, window=300), dm.moe(experts=16, top=4, ff=64, shared=96))],
                width=128, vocab=200),
    "many heads": dict(layers=[(dm.talking(heads=36, kv_heads=4, dim=24, vdim=40, rot=16), None),
                               (dm.latent(heads=40, dim=16, rot=8, vdim=24, rank=64, q_rank=48, window=90), dm.dense(128))], width=192, vocab=100),
    "wide rows": dict(layers=[(dm.talking(heads=10, kv_heads=5, dim=128, vdim=128, rot=32, scale=0.1), None),
                              (dm.talking(heads=8, kv_heads=8, dim=64, vdim=72, rot=64, scale=0.1), dm.dense(64))], width=128, vocab=90),
}
SINGLE = {
    "mixed heads": dict(layers=[(dm.talking(heads=4, kv_heads=2, dim=64, vdim=64, rot=32), None)]),
    "mixed heads odd": dict(layers=[(dm.talking(heads=3, kv_heads=1, dim=33, vdim=17, rot=20), None)]),
    "latent": dict(layers=[(dm.latent(heads=4, dim=32, rot=16, vdim=40, rank=96, q_rank=40, window=48), None)]),
    "latent odd": dict(layers=[(dm.latent(heads=3, dim=30, rot=14, vdim=19, rank=45, q_rank=33, window=65), None)]),
    "dense": dict(layers=[(dm.latent(heads=2), dm.dense(128))]),
    "experts": dict(layers=[(dm.talking(heads=2, kv_heads=1), dm.moe(experts=8, top=3, ff=128, shared=128))]),
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
@pytest.mark.parametrize("window", [63, 64, 65, 128, 129, 300])
def test_keys_at_the_edges_of_the_window(window, dtype, tmp_path):
    """One key carries the whole answer, just inside and just outside the window: prompts, portions and decoding."""
    n = 420
    for at in (n - 1 - window, n - window, n - 2):
        _pointer(dm.latent(heads=4, dim=64, rot=32, vdim=64, rank=64, q_rank=40, window=window), at, n, dtype, tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim", [(4, 2, 64), (6, 3, 128)])
def test_far_keys_of_mixed_heads(heads, kv_heads, dim, dtype, tmp_path):
    for at in (0, 15, 64, 127, 128, 255, 256, 417):
        _pointer(dm.talking(heads=heads, kv_heads=kv_heads, dim=dim, vdim=64, rot=32), at, 420, dtype, tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["wide", "wide rows"])
def test_pages_with_old_contents(name, dtype, tmp_path):
    cfg, w, path = _model(name, dtype, tmp_path)
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


@pytest.mark.parametrize("impl", [1, 2, 3])
@pytest.mark.parametrize("name", ["wide", "mid", "many heads"])
def test_other_forms_of_attention_agree(name, impl, tmp_path, monkeypatch):
    """Forms that are not the first choice: 1 without tensor cores, 2 the form of decode batches also in prefill, 3 the same on
    mma.sync (latent attention)."""
    from fastcache_b200.ops import hybrid
    monkeypatch.setattr(hybrid, "LATENT_IMPL", impl)
    monkeypatch.setattr(hybrid, "TALK_IMPL", min(impl, 2))
    cfg, w, path = _model(name, "bfloat16", tmp_path)
    prompts = {"a": dm.tokens(190, cfg["vocab"], 1)}
    llm = dm.engine(path, "cuda", "bfloat16", enforce_eager=True)
    _check(dm.feed(llm, prompts, [[("a", 170)], [("a", 18)], [("a", 1)], [("a", 1)]])["a"],
           dm.expected(cfg, w, prompts)["a"], "bfloat16", "other forms")
    llm.exit()


def test_long_context_decode_with_splits_and_large_prompts(tmp_path):
    cfg, w, path = _model("mid", "bfloat16", tmp_path)
    n = 1500
    prompts = {"a": dm.tokens(n, cfg["vocab"], 1), "b": dm.tokens(n // 3, cfg["vocab"], 2)}
    want = {i: oracle.forward(cfg, w, t, torch.float32)[0] for i, t in prompts.items()}
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


def _softmax(s, sink):
    if sink is not None:
        s = torch.cat([s, sink.double()[:, None].expand(s.shape[0], 1) if s.dim() == 2 else sink.double()[:, None, None].expand(-1, s.shape[1], 1)], -1)
        return torch.softmax(s, -1)[..., :-1]
    return torch.softmax(s, -1)


@pytest.mark.parametrize("impl", [0, 1])
@pytest.mark.parametrize("H,G,D,V,page,window,sink", [(32, 2, 128, 128, 64, 0, False), (8, 2, 64, 40, 16, 0, False), (33, 3, 40, 24, 8, 100, True),
                                                      (32, 8, 128, 128, 64, 0, True), (6, 6, 64, 72, 32, 65, False), (16, 4, 128, 128, 64, 700, False),
                                                      (12, 1, 128, 96, 256, 1, True), (48, 4, 96, 128, 64, 64, True)])
def test_attention_over_rows_with_several_value_heads(H, G, D, V, page, window, sink, impl):
    from fastcache_b200.ops.loader import ext
    ctx = torch.tensor([1, 700, 0, 127, 128, 129, 1030, 2500, 64], dtype=torch.int32, device="cuda")
    pages, B, v_col = -(-2500 // page), ctx.numel(), G * D + 8
    pool = _rnd(B * pages, page, v_col + G * V, seed=H)
    bt = torch.randperm(B * pages, device="cuda", generator=torch.Generator(device="cuda").manual_seed(H)).int().view(B, pages)
    q = _rnd(B, H, G * D, seed=1)
    sinks = _rnd(H, scale=3.0, dtype=torch.float32, seed=2) if sink else None
    gate = torch.rand(B, H, device="cuda") if sink else None
    for scale in (0.02, 0.4, 8.0):            # the last: scores hundreds of e-folds apart, one row takes all
        got = ext().latent_decode_rows(q, pool, bt, ctx, V, scale, impl, v_col, G, window, sinks, gate).double()
        for i, n in enumerate(ctx.tolist()):
            first = max(0, n - window) if window else 0
            rows = pool[bt[i].long()].reshape(-1, pool.shape[-1])[first:n].double()
            p = _softmax(q[i].double() @ rows[:, :G * D].T * scale, sinks)
            v = rows[:, v_col:].view(n - first, G, V).repeat_interleave(H // G, 1)
            want = torch.einsum("hj,jhv->hv", p, v) * (1 if gate is None else gate[i].double()[:, None])
            assert (got[i] - want).abs().max().item() < 0.04, (scale, n)
    assert ext().read_status(0) == 0


@pytest.mark.parametrize("impl", [0, 1, 3])
@pytest.mark.parametrize("H,rank,R,page,window", [(32, 512, 64, 64, 600), (5, 128, 32, 16, 33), (20, 256, 64, 256, 128), (3, 64, 16, 8, 1)])
def test_absorbed_attention_with_window_sink_and_gate(H, rank, R, page, window, impl):
    from fastcache_b200.ops.loader import ext
    ctx = torch.tensor([1, 700, 0, 127, 128, 129, 1030, 2500, 64], dtype=torch.int32, device="cuda")
    pages, B = -(-2500 // page), ctx.numel()
    pool = _rnd(B * pages, page, rank + R, seed=H)
    bt = torch.randperm(B * pages, device="cuda", generator=torch.Generator(device="cuda").manual_seed(H)).int().view(B, pages)
    q, sinks, gate = _rnd(B, H, rank + R, seed=1), _rnd(H, scale=3.0, dtype=torch.float32, seed=2), torch.rand(B, H, device="cuda")
    for scale in (0.02, 0.5, 8.0):
        got = ext().latent_decode_rows(q, pool, bt, ctx, rank, scale, impl, 0, 1, window, sinks, gate).double()
        for i, n in enumerate(ctx.tolist()):
            rows = pool[bt[i].long()].reshape(-1, pool.shape[-1])[max(0, n - window):n].double()
            want = _softmax(q[i].double() @ rows.T * scale, sinks) @ rows[:, :rank] * gate[i].double()[:, None]
            assert (got[i] - want).abs().max().item() < 0.04, (scale, n)
    assert ext().read_status(0) == 0


@pytest.mark.parametrize("H,G,D,R,V,window,sink", [(4, 2, 0, 64, 64, 0, False), (3, 1, 0, 256, 128, 0, False), (6, 1, 0, 40, 24, 0, False),
                                                   (4, 1, 0, 136, 72, 0, False), (16, 2, 0, 192, 128, 0, False), (8, 2, 0, 256, 128, 0, False), (6, 3, 0, 336, 80, 0, False),
                                                   (4, 4, 0, 512, 128, 0, True), (4, 1, 0, 384, 56, 50, False), (10, 5, 0, 640, 128, 0, False),
                                                   (8, 8, 0, 1024, 64, 129, True), (3, 3, 128, 64, 128, 100, True), (2, 2, 40, 24, 16, 1, True),
                                                   (2, 2, 128, 64, 128, 128, False)])
def test_prefill_over_gathered_rows(H, G, D, R, V, window, sink):
    """Keys of their own and shared ones, value heads, windows, sinks: portions behind a past, of unequal requests."""
    from fastcache_b200.ops.loader import ext
    q_lens, kv_lens = (300, 1, 129, 2, 64), (300, 257, 400, 2, 500)
    cu_q, cu_kv = (torch.tensor([0] + list(torch.tensor(x).cumsum(0)), dtype=torch.int32, device="cuda") for x in (q_lens, kv_lens))
    T, N = sum(q_lens), sum(kv_lens)
    q, kv, rot = _rnd(T, H, D + R, seed=1), _rnd(N, H * D + G * V, seed=2), _rnd(N, R, seed=3)
    sinks = _rnd(H, scale=2.0, dtype=torch.float32, seed=4) if sink else None
    for scale in (0.05, 1.0):
        got = ext().latent_prefill_rows(q, kv, rot, None, cu_q, cu_kv, D, V, scale, max(q_lens), G, window, sinks).double()
        for b, (n, m) in enumerate(zip(q_lens, kv_lens)):
            a, c = int(cu_q[b]), int(cu_kv[b])
            k = kv[c:c + m, :H * D].view(m, H, D).double()
            v = kv[c:c + m, H * D:].view(m, G, V).repeat_interleave(H // G, 1).double()
            s = torch.einsum("ihd,jhd->hij", q[a:a + n, :, :D].double(), k) + torch.einsum("ihr,jr->hij", q[a:a + n, :, D:].double(), rot[c:c + m].double())
            i, j = torch.arange(m - n, m, device="cuda")[:, None], torch.arange(m, device="cuda")[None]
            seen = (j <= i) & ((i - j < window) if window else True)
            want = torch.einsum("hij,jhv->ihv", _softmax((s * scale).masked_fill(~seen, float("-inf")), sinks), v).reshape(n, H * V)
            assert (got[a:a + n] - want).abs().max().item() < 0.05, (scale, b)
    assert ext().read_status(0) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E,top", [(1, 6, 2), (70, 16, 4), (256, 40, 3), (700, 5, 5), (1000, 130, 1)])
def test_routing_by_logit(T, E, top, dtype):
    from fastcache_b200.ops import hybrid, reference_hybrid as ref
    from fastcache_b200.utils.context import Context
    h, weight = _rnd(T, 64, dtype=dtype, seed=E), torch.zeros(-(-(E + 1) // 8) * 8, 64, device="cuda", dtype=dtype)
    weight[:E + 1] = _rnd(E + 1, 64, scale=0.3, dtype=dtype, seed=2)
    bias = 4 * torch.randperm(E, device="cuda").float() / 2       # no close calls among the chosen
    bias += 0.01 * torch.randn(E, device="cuda")
    (row_of, plan), mix, factor = hybrid.route_by_logit(h, weight, bias, top, True, Context(is_prefill=True))
    ids, w, f = ref.route_by_logit(h.float().cpu() @ weight.float().cpu().T, bias.cpu(), top, True)
    token = plan[len(plan) - T * top:].cpu()
    assert torch.equal(token[row_of.flatten().long().cpu()], torch.arange(T).repeat_interleave(top).int())
    first = plan[:E + 1].cpu()
    got = torch.bucketize(row_of.cpu().flatten(), first, right=True).view(T, top) - 1
    same = (got == ids).all(1)
    assert same.float().mean() > 0.97
    assert (mix.cpu() - w)[same].abs().max() < 2e-3 and (factor.cpu() - f).abs().max() < 2e-3
    assert (mix.sum(1) - 1).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,width,ff", [(1, 64, 24), (37, 96, 77), (300, 128, 256), (520, 64, 50)])
def test_xielu_of_a_product(T, width, ff, dtype):
    from fastcache_b200.ops import hybrid
    h, w = _rnd(T, width, dtype=dtype), torch.zeros(-(-ff // 8) * 8, width, device="cuda", dtype=dtype)
    w[:ff] = _rnd(ff, width, scale=2 * width ** -0.5, dtype=dtype, seed=1)
    p, q = torch.tensor(0.3).double(), torch.tensor(-1.1).double()
    coef = torch.tensor([oracle.softplus(p), 0.5 + oracle.softplus(q)], device="cuda").float()
    got = hybrid.linear_xielu(h, w, coef, ff)
    want = oracle.xielu(h.double().cpu() @ w[:ff].double().cpu().T, p, q)
    err = (got[:, :ff].double().cpu() - want).abs() / (1 + want.abs())
    assert err.max() < (2e-2 if dtype == torch.bfloat16 else 1e-5) and got[:, ff:].abs().sum() == 0
