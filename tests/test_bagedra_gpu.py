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
                 width=256, ff=320, vocab=520),
    "mid": dict(mixers=[bm.gla(heads=2, dim=32, vdim=64, tau=2.0), bm.latent(heads=20, dim=96, rot=24, vdim=64, rank=128),
                        bm.delta(heads=2, kv_heads=1, dim=64, vdim=128)], width=128, ff=96, vocab=200),
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
