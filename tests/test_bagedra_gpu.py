"""Bagedra on a CUDA device: the engine's kernels in bf16 and fp32 against the plain implementation."""
import pytest
import torch

import bagedra_models as bm

pytestmark = pytest.mark.gpu

LIMIT = {"bfloat16": 0.2, "float32": 2e-4}            # worst position
MEAN_LIMIT = {"bfloat16": 0.02, "float32": 2e-5}      # all positions

# (mixers, other settings): sizes for the tensor-core forms and sizes that only the general kernels take
MODELS = {
    "general": dict(mixers=[bm.delta(), bm.latent(), bm.gla(), bm.latent(kv_from=1)]),
    "odd": dict(mixers=[bm.latent(dim=12, rot=6, vdim=10, rank=20), bm.gla(heads=1, dim=7, vdim=9, tau=1.0),
                        bm.delta(heads=2, kv_heads=2, dim=5, vdim=130, conv=1),
                        bm.latent(heads=1, dim=3, rot=6, vdim=11, rank=20, kv_from=0)],
                width=61, ff=45, vocab=77, no_mlp=(1, 3)),
    "wide": dict(mixers=[bm.latent(heads=4, dim=128, rot=64, vdim=128, rank=256), bm.gla(heads=2, dim=128, vdim=128),
                         bm.delta(heads=4, kv_heads=2, dim=128, vdim=128, conv=4),
                         bm.latent(heads=8, dim=64, rot=64, vdim=96, rank=256, kv_from=0),
                         bm.gla(heads=2, dim=64, vdim=256), bm.delta(heads=2, kv_heads=1, dim=96, vdim=64)],
                 width=256, ff=384, vocab=520),
    "mid": dict(mixers=[bm.gla(heads=2, dim=32, vdim=64, tau=2.0), bm.latent(heads=20, dim=96, rot=24, vdim=64, rank=128),
                        bm.delta(heads=2, kv_heads=1, dim=64, vdim=128)], width=128, ff=96, vocab=200),
    "heads": dict(mixers=[bm.latent(heads=40, dim=32, rot=32, vdim=32, rank=128), bm.delta(heads=12, kv_heads=3, dim=16, vdim=16),
                          bm.latent(heads=70, dim=16, rot=32, vdim=16, rank=128, kv_from=0), bm.gla(heads=12, dim=16, vdim=16)],
                  width=192, ff=256, vocab=100),
}
SINGLE = {
    "latent": [bm.latent(heads=2, dim=64, rot=32, vdim=64, rank=64)],
    "latent odd": [bm.latent(heads=2, dim=33, rot=10, vdim=13, rank=37)],
    "gla": [bm.gla(heads=2, dim=48, vdim=80, tau=4.0)],
    "gla strong decay": [bm.gla(heads=2, dim=48, vdim=32, tau=0.25)],
    "delta": [bm.delta(heads=4, kv_heads=2, dim=80, vdim=48, conv=4)],
    "delta six taps": [bm.delta(heads=2, kv_heads=1, dim=24, vdim=40, conv=6)],
}


def _model(name, tmp_path):
    cfg = bm.config(**MODELS[name])
    w = bm.weights(cfg, seed=len(name))
    return cfg, w, bm.save(tmp_path / name, cfg, w)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_portions_decode_and_mixed_batches(name, dtype, tmp_path):
    cfg, w, path = _model(name, tmp_path)
    prompts = {"a": bm.tokens(301, cfg["vocab"], 1), "b": bm.tokens(150, cfg["vocab"], 2),
               "c": bm.tokens(17, cfg["vocab"], 3), "d": bm.tokens(1, cfg["vocab"], 4)}
    want = bm.expected(cfg, w, prompts)
    whole = [[(i, len(t))] for i, t in prompts.items()]
    together = [[(i, len(t)) for i, t in prompts.items()]]
    cut = [[("a", 2), ("b", 65)], [("a", 64), ("d", 1)], [("b", 1)], [("a", 130), ("b", 1), ("c", 2)],
           [("c", 1), ("b", 1)], [("b", 63), ("a", 1), ("c", 1)], [("a", 60), ("b", 2), ("c", 13)]] + \
          [[("a", 1), ("b", 1)]] * 17 + [[("a", 1)]] * 27
    llm = bm.engine(path, "cuda", dtype)
    for schedule in (whole, together, cut):
        got = bm.feed(llm, prompts, schedule)
        for i in prompts:
            worst, mean = bm.errors(got[i], want[i])
            assert worst < LIMIT[dtype] and mean < MEAN_LIMIT[dtype], (i, schedule[0], worst, mean)
    llm.exit()


def _check(got, want, dtype, what):
    worst, mean = bm.errors(got, want)
    assert worst < LIMIT[dtype] and mean < MEAN_LIMIT[dtype], (what, worst, mean)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_in_portions_of_several_sizes(name, dtype, tmp_path):
    cfg = bm.config(SINGLE[name], width=96, ff=64, vocab=90)
    w = bm.weights(cfg, seed=11)
    llm = bm.engine(bm.save(tmp_path / "m", cfg, w), "cuda", dtype)
    prompts = {"a": bm.tokens(206, cfg["vocab"], 5)}
    want = bm.expected(cfg, w, prompts)["a"]
    for sizes in ([206], [2] * 103, [64, 64, 64, 14], [63, 1, 65, 1, 76], [30, 1, 25, 150], [130] + [1] * 76):
        got = bm.feed(llm, prompts, [[("a", n)] for n in sizes])["a"]
        _check(got, want, dtype, sizes[:5])
    llm.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_single_far_key_at_page_and_tile_borders(dtype, tmp_path):
    """One key carries the whole answer: prompts, portions and decoding, pages of 16 and of 64 tokens."""
    n = 420
    for at in (0, 1, 15, 16, 63, 64, 127, 128, 129, 255, 256, 383, 384, 417):
        cfg, w, prompt = bm.pointer_model(at, n, bm.latent(heads=2, dim=64, rot=32, vdim=64, rank=64))
        want = bm.oracle.forward(cfg, w, prompt)[0]
        path = bm.save(tmp_path / f"m{at}", cfg, w)
        llm = bm.engine(path, "cuda", dtype, page=64 if at % 2 else 16, enforce_eager=True)
        for cut in ([n], [n - 1, 1], [at + 1, n - at - 3, 2], [256, 129, n - 385]):
            got = bm.feed(llm, {"a": prompt}, [[("a", c)] for c in cut if c])["a"]
            worst, _ = bm.errors(got[-1:], want[-1:])
            assert worst < (0.05 if dtype == "bfloat16" else 2e-4), (at, cut, worst)
        llm.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_with_old_contents(dtype, tmp_path):
    cfg, w, path = _model("wide", tmp_path)
    llm = bm.engine(path, "cuda", dtype, max_tokens=20 * bm.PAGE, requests=2)
    for c in llm.model_runner.cache_layout:
        for name in c.state:
            getattr(c.module, name).fill_(1e3)
        if c.row_width:
            c.module.rows.fill_(1e3)
    for k in range(4):
        prompts = {f"x{k}": bm.tokens(130 + k, cfg["vocab"], k), f"y{k}": bm.tokens(90 - 20 * k, cfg["vocab"], 50 + k)}
        want = bm.expected(cfg, w, prompts)
        a, b = prompts
        n, m = len(prompts[a]), len(prompts[b])
        got = bm.feed(llm, prompts, [[(b, 1)], [(a, 100), (b, 3)], [(a, n - 103), (b, 1)], [(b, m - 8), (a, 1)],
                                     [(a, 1), (b, 1)], [(a, 1), (b, 1)], [(b, 1)]])
        for i in prompts:
            _check(got[i], want[i], dtype, i)
    llm.exit()


@pytest.mark.parametrize("impl", [1, 2, 3])
@pytest.mark.parametrize("name", ["wide", "heads"])
def test_other_forms_of_latent_attention_agree(name, impl, tmp_path, monkeypatch):
    """Forms that are not the first choice: 1 without tensor cores, 2 absorbed attention also in prefill,
    3 the same on mma.sync."""
    from fastcache_b200.ops import hybrid
    monkeypatch.setattr(hybrid, "LATENT_IMPL", impl)
    cfg, w, path = _model(name, tmp_path)
    prompts = {"a": bm.tokens(90, cfg["vocab"], 1)}
    llm = bm.engine(path, "cuda", "bfloat16", enforce_eager=True)
    _check(bm.feed(llm, prompts, [[("a", 70)], [("a", 18)], [("a", 1)], [("a", 1)]])["a"],
           bm.expected(cfg, w, prompts)["a"], "bfloat16", "general")
    llm.exit()


def _absorbed(q, pool, bt, ctx, rank, scale):
    out = []
    for i, n in enumerate(ctx.tolist()):
        rows = pool[bt[i].long()].reshape(-1, pool.shape[-1])[:n, :q.shape[-1]].double()
        s = (q[i].double() @ rows.T) * scale
        out.append(torch.softmax(s, -1) @ rows[:, :rank] if n else torch.zeros(q.shape[1], rank, device=q.device))
    return torch.stack([o.double() for o in out])


@pytest.mark.parametrize("impl", [0, 1, 3])
@pytest.mark.parametrize("H,rank,R,page", [(32, 512, 64, 64), (5, 128, 32, 16), (70, 256, 64, 256), (33, 64, 32, 8),
                                           (16, 320, 64, 32), (1, 16, 8, 128)])
def test_absorbed_attention_over_pages(H, rank, R, page, impl):
    from fastcache_b200.ops.loader import ext
    g = torch.Generator(device="cuda").manual_seed(H)
    ctx = torch.tensor([1, 700, 0, 127, 128, 129, 1030, 2500, 64], dtype=torch.int32, device="cuda")
    pages = -(-2500 // page)
    B = ctx.numel()
    pool = torch.randn(B * pages, page, rank + R, device="cuda", generator=g).bfloat16()
    bt = torch.randperm(B * pages, device="cuda", generator=g).int().view(B, pages)
    q = torch.randn(B, H, rank + R, device="cuda", generator=g).bfloat16()
    for scale in (0.02, 0.5, 8.0):            # the last: scores hundreds of e-folds apart, one row takes all
        got = ext().latent_decode_rows(q, pool, bt, ctx, rank, scale, impl).double()
        want = _absorbed(q, pool, bt, ctx, rank, scale)
        err = (got - want).abs().max().item()
        assert err < 0.04, (scale, err)
    assert ext().read_status(0) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_steps_that_read_nothing_back(dtype, tmp_path):
    """Decode steps whose logits nobody asks for, one after another, then one that is asked for."""
    from fastcache_b200.engine.replay import TokenReplay
    cfg, w, path = _model("general", tmp_path)
    llm = bm.engine(path, "cuda", dtype)
    replay = TokenReplay(llm)
    for k, n in enumerate((97, 23, 140, 64)):
        toks = bm.tokens(n, cfg["vocab"], k)
        name = f"r{k}"
        replay.step([{"id": name, "tokens": toks[:4], "want": []}])
        for t in toks[4:-1]:
            replay.step([{"id": name, "tokens": [t], "want": []}])
        got = replay.step([{"id": name, "tokens": toks[-1:], "want": [0]}], [name])
        assert bm.errors(got, bm.oracle.forward(cfg, w, toks)[0][-1:])[0] < LIMIT[dtype], n
    llm.exit()


def test_long_context_decode_with_splits(tmp_path):
    cfg, w, path = _model("mid", tmp_path)
    n = 1500
    prompts = {"a": bm.tokens(n, cfg["vocab"], 1), "b": bm.tokens(n // 3, cfg["vocab"], 2)}
    want = bm.expected(cfg, w, prompts)
    llm = bm.engine(path, "cuda", "bfloat16", max_tokens=4096)
    got = bm.feed(llm, prompts, [[("a", n - 40), ("b", n // 3 - 40)]] + [[("a", 1), ("b", 1)]] * 40)
    for i in prompts:
        _check(got[i], want[i], "bfloat16", i)
    llm.exit()


@pytest.mark.parametrize("name", ["general", "wide"])
def test_generation_matches_between_graph_and_eager_and_single_requests(name, tmp_path):
    from fastcache_b200 import SamplingParams
    cfg, w, path = _model(name, tmp_path)
    prompts = [bm.tokens(n, cfg["vocab"], n) for n in (70, 3, 33, 129, 1)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    outs = []
    for kw in (dict(enforce_eager=True), dict(), dict(max_num_batched_tokens=40, chunked_prefill_tokens=8)):
        llm = bm.engine(path, "cuda", "float32", **kw)
        outs.append([o["token_ids"] for o in llm.generate(prompts, sp)])
        llm.exit()
    assert outs[0] == outs[1] == outs[2]
    seq = prompts[0] + outs[0][0]
    logits = bm.oracle.forward(cfg, w, seq)[0]
    assert logits[len(prompts[0]) - 1:-1].argmax(-1).tolist() == outs[0][0]
