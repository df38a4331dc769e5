"""Darusun through the engine on CPU (32-bit): cache, scheduler and loader against the plain statements."""
import json
import math
import subprocess
import sys

import numpy as np
import pytest
import torch

import darusun_models as dm
import darusun_oracle as oracle
from fastcache_b200 import SamplingParams
from fastcache_b200.engine.replay import TokenReplay

MIX = dict(layers=[(dm.talking(heads=4, kv_heads=2, dim=12, vdim=10, rot=8), dm.moe(experts=6, top=2, ff=20, shared=14)),
                   (dm.latent(heads=3, dim=10, rot=6, vdim=8, rank=12, q_rank=14, window=18), dm.dense(24)),
                   (dm.talking(heads=4, kv_heads=2, dim=12, vdim=10, rot=8, scale=0.5, kv_from=0), None),
                   (dm.latent(heads=2, dim=8, rot=4, vdim=12, rank=10, q_rank=9, window=7), dm.moe(experts=5, top=3, ff=12, shared=20)),
                   (dm.talking(heads=6, kv_heads=3, dim=8, vdim=6, rot=4, base=100.0), dm.dense(30))],
           width=40, vocab=60)
SINGLE = {
    "mixed heads": dict(layers=[(dm.talking(), None)]),
    "mixed heads, one key head": dict(layers=[(dm.talking(heads=5, kv_heads=1, dim=9, vdim=7, rot=6), None)]),
    "mixed heads, a key head each": dict(layers=[(dm.talking(heads=3, kv_heads=3, dim=10, vdim=10, rot=10), dm.dense(9))]),
    "one head": dict(layers=[(dm.talking(heads=1, kv_heads=1, dim=8, vdim=13, rot=2), None)]),
    "large scale": dict(layers=[(dm.talking(scale=1.0), None)]),
    "shared rows": dict(layers=[(dm.talking(), None), (dm.latent(), None), (dm.talking(scale=0.3, kv_from=0), dm.dense()),
                                (dm.talking(kv_from=0), None)]),
    "latent": dict(layers=[(dm.latent(), None)]),
    "latent, window of one": dict(layers=[(dm.latent(window=1), None)]),
    "latent, window of a page": dict(layers=[(dm.latent(heads=1, dim=6, rot=8, vdim=20, rank=40, q_rank=5, window=16), dm.dense(20))]),
    "latent, window past the prompt": dict(layers=[(dm.latent(window=500, scale=0.1), None)]),
    "dense": dict(layers=[(dm.latent(), dm.dense(50))]),
    "experts": dict(layers=[(dm.latent(), dm.moe())]),
    "one expert of many": dict(layers=[(dm.talking(), dm.moe(experts=12, top=1, ff=12, shared=40))]),
    "all experts": dict(layers=[(dm.talking(), dm.moe(experts=3, top=3, ff=11, shared=5))]),
    "multiplier of one": dict(layers=[(dm.talking(), dm.dense()), (dm.latent(), dm.moe())], mult=1.0),
}
TOL = 2e-5


def _model(tmp_path, spec, seed=0, **kw):
    cfg = dm.config(**dict(spec, **kw))
    w = dm.weights(cfg, seed=seed)
    return cfg, w, dm.save(tmp_path / "m", cfg, w)


def _cuts(n, sizes):
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_whole_and_in_portions(name, tmp_path):
    cfg, w, path = _model(tmp_path, SINGLE[name], seed=3)
    prompts = {"a": dm.tokens(53, cfg["vocab"], 5)}
    want = dm.expected(cfg, w, prompts)
    llm = dm.engine(path, "cpu", "float32")
    for sizes in ([53], [1], [2], [20, 1, 1, 3], [16, 17, 15]):
        got = dm.feed(llm, prompts, [[("a", n)] for n in _cuts(53, sizes)])
        assert dm.errors(got["a"], want["a"])[0] < TOL, sizes


def test_the_plain_statements_by_hand():
    """Small numbers whose results are known."""
    rot = dict(base=100.0, dims=4)
    x, at = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]]).double(), torch.tensor([2])
    a, b = 2.0, 0.2                                          # angles of the two pairs
    half = oracle.rotate_half(x, at, rot)[0, 0]
    pairs = oracle.rotate_pairs(x, at, rot)[0, 0]
    assert torch.allclose(half, torch.tensor([math.cos(a) - 3 * math.sin(a), 2 * math.cos(b) - 4 * math.sin(b),
                                              3 * math.cos(a) + math.sin(a), 4 * math.cos(b) + 2 * math.sin(b), 5.0]).double())
    assert torch.allclose(pairs, torch.tensor([math.cos(a) - 2 * math.sin(a), 2 * math.cos(a) + math.sin(a),
                                               3 * math.cos(b) - 4 * math.sin(b), 4 * math.cos(b) + 3 * math.sin(b), 5.0]).double())
    s = torch.tensor([1.0, 2.0])[:, None, None].expand(2, 1, 1)
    assert oracle.mix_heads(s, torch.tensor([[1.0, 10.0], [0.5, 0.0]])).flatten().tolist() == [21.0, 0.5]
    assert oracle.sliding_window(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    p = oracle.softmax(torch.zeros(1, 1, 3), torch.tensor([[True, True, False]]), torch.tensor([math.log(2.0)]))
    assert torch.allclose(p.flatten(), torch.tensor([0.25, 0.25, 0.0]))
    z, zero = torch.tensor([2.0, -1.0, 0.0]).double(), torch.tensor(0.0).double()
    ln2 = math.log(2.0)
    assert torch.allclose(oracle.xielu(z, zero, zero), torch.tensor([4 * ln2 + 1, (0.5 + ln2) * math.exp(-1) - 0.5, 0.0]).double())
    got = oracle.route(torch.tensor([0.0, 1.0, -5.0, 1.0 + ln2]), 2)
    assert sorted(got) == [1, 3] and abs(got[3] - 2 / 3) < 1e-6


def test_scores_of_mixed_heads_are_scores_of_wide_queries():
    g = torch.Generator().manual_seed(0)
    H, G, D, T = 6, 3, 5, 7
    q, k = torch.randn(T, H, D, generator=g), torch.randn(T, G, D, generator=g)
    talk = torch.randn(H, H, generator=g)
    want = oracle.mix_heads(torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)), talk)
    wide = torch.stack([torch.einsum("hg,igd->ihd", talk[:, u * H // G:(u + 1) * H // G], q[:, u * H // G:(u + 1) * H // G])
                        for u in range(G)], 2)
    assert torch.allclose(torch.einsum("ihc,jc->hij", wide.flatten(2), k.flatten(1)), want, atol=1e-4)


def _changes():
    def cfg(path, value):
        def f(c, w):
            for key in path[:-1]:
                c = c[key]
            c[path[-1]] = value
        return f

    def tensor(name, change):
        return lambda c, w: w.update({name: change(w[name])})

    def swap(a, b):
        def f(c, w):
            w[a], w[b] = w[b], w[a]
        return f

    out = {"window": cfg(("layers", 1, "mixer", "mask", "size"), 19), "short window": cfg(("layers", 3, "mixer", "mask", "size"), 6),
           "rotated dimensions": cfg(("layers", 4, "mixer", "rot", "dims"), 6), "base": cfg(("layers", 1, "mixer", "rot", "base"), 3300.0),
           "scale": cfg(("layers", 2, "mixer", "scale"), 0.49), "latent scale": cfg(("layers", 3, "mixer", "scale"), 0.3),
           "top": cfg(("layers", 3, "mlp", "router", "top"), 2), "multiplier": cfg(("residual_mult",), 0.59), "eps": cfg(("norm", "eps"), 1e-2),
           "own rows": lambda c, w: (c["layers"][2]["mixer"].pop("kv_from"), w.update({f"l2.mix.{n}": w[f"l0.mix.{n}"] for n in "kv"})),
           "other rows": lambda c, w: w.update({"l0.mix.v": w["l0.mix.v"].roll(1, 0)}),
           "talk": tensor("l0.mix.talk", lambda t: torch.eye(4)), "talk, from and to": tensor("l2.mix.talk", lambda t: t.T),
           "sink": tensor("l1.mix.sink", lambda t: t - 30), "gate": tensor("l3.mix.g", lambda t: 0 * t),
           "query norm": tensor("l1.mix.dq.norm", torch.ones_like), "latent norm": tensor("l3.mix.dkv.norm", torch.ones_like),
           "act": swap("l1.mlp.act", "l4.mlp.act"), "act, p and q": tensor("l4.mlp.act", lambda t: t.flip(0)),
           "router bias": tensor("l0.mlp.router.b", lambda t: 0 * t), "shared gate": tensor("l3.mlp.shared.sg", lambda t: 0 * t),
           "shared expert": tensor("l0.mlp.shared.up", lambda t: 0 * t)}
    for name in ("l0.norm1", "l1.norm2", "l2.norm1", "l3.norm2", "final.norm"):
        out[name] = tensor(name, torch.ones_like)
    return out


@pytest.mark.parametrize("change", list(_changes()))
def test_the_random_models_show_a_fault(change):
    """Every mechanism of the models above leaves a trace in the logits: change it in the plain statements and look."""
    cfg = dm.config(**MIX)
    w = dm.weights(cfg)
    prompt = dm.tokens(50, cfg["vocab"], 1)
    want = oracle.forward(cfg, w, prompt)[0]
    c, v = json.loads(json.dumps(cfg)), dict(w)
    _changes()[change](c, v)
    assert dm.errors(oracle.forward(c, v, prompt)[0][-20:], want[-20:])[0] > 100 * TOL


def test_unequal_requests_together_and_alone(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    prompts = {c: dm.tokens(n, cfg["vocab"], n) for c, n in zip("abcd", (45, 1, 33, 7))}
    want = dm.expected(cfg, w, prompts)
    schedule = [[("a", 3), ("c", 17)], [("b", 1), ("c", 1), ("a", 14)], [("d", 2), ("a", 1)], [("c", 15), ("d", 1)],
                [("a", 25), ("d", 4)]] + [[("a", 1)], [("a", 1)]]
    got = dm.feed(dm.engine(path, "cpu", "float32"), prompts, schedule)
    for i in prompts:
        assert dm.errors(got[i], want[i])[0] < TOL, i


def fill_caches(llm, value):
    for c in llm.model_runner.cache_layout:
        c.module.rows.fill_(value)


def test_pages_are_used_again(tmp_path):
    """A pool with room for two requests of three pages, filled with junk first: many requests in turn."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = dm.engine(path, "cpu", "float32", max_tokens=6 * dm.PAGE, requests=2)
    fill_caches(llm, 100.0)
    replay = TokenReplay(llm)
    tables = set()
    for k in range(6):
        prompts = {f"x{k}": dm.tokens(35 + k, cfg["vocab"], k), f"y{k}": dm.tokens(20 + k, cfg["vocab"], 50 + k)}
        want = dm.expected(cfg, w, prompts)
        names = list(prompts)
        for n in (names if k % 2 else names[::-1]):
            replay.step([{"id": n, "tokens": prompts[n][:10], "want": []}])
        tables |= {tuple(replay.live[n].block_table) for n in names}
        got = replay.step([{"id": n, "tokens": prompts[n][10:], "want": [len(prompts[n]) - 11]} for n in names], names)
        for i, n in enumerate(names):
            assert dm.errors(got[i:i + 1], want[n][-1:])[0] < TOL
    assert len(tables) > 2
    llm.scheduler.block_manager.check_invariants([])


def _pointer(spec, at, n, visible, tmp_path):
    cfg, w, prompt = dm.pointer_model(spec, at, n)
    want = oracle.forward(cfg, w, prompt)[0]
    without = list(prompt)
    without[at] = 5
    seen = dm.errors(oracle.forward(cfg, w, without)[0][-1:], want[-1:])[0]
    assert seen > 0.3 if visible else seen < 1e-6
    llm = dm.engine(dm.save(tmp_path / f"m{at}", cfg, w), "cpu", "float32")
    for cut in ([n], [n - 1, 1], [at + 1, n - at - 2, 1], [32, 31, n - 63]):
        got = dm.feed(llm, {"a": prompt}, [[("a", c)] for c in cut if c])
        assert dm.errors(got["a"], want)[0] < TOL, (at, cut)


@pytest.mark.parametrize("window", [15, 16, 17, 32, 40])
def test_keys_at_the_edges_of_the_window(window, tmp_path):
    """One key carries the whole answer: just inside the window it decides the last logits, just outside it is not there."""
    n = 70
    spec = dm.latent(heads=3, dim=12, rot=6, vdim=16, rank=20, q_rank=16, window=window)
    for at in (n - 1 - window, n - window, n - 2, 0):
        _pointer(spec, at, n, at >= n - window, tmp_path)


@pytest.mark.parametrize("at", [0, 1, 15, 16, 31, 32, 67, 68])
def test_far_keys_of_mixed_heads(at, tmp_path):
    _pointer(dm.talking(heads=4, kv_heads=2, dim=16, vdim=12, rot=6), at, 70, True, tmp_path)


def test_long_decoding(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    prompts = {"a": dm.tokens(150, cfg["vocab"], 1), "b": dm.tokens(140, cfg["vocab"], 2)}
    got = dm.feed(dm.engine(path, "cpu", "float32"), prompts, [[("a", 12), ("b", 2)]] + [[("a", 1), ("b", 1)]] * 138)
    want = dm.expected(cfg, w, prompts)
    assert all(dm.errors(got[i], want[i])[0] < TOL for i in prompts)


@pytest.mark.parametrize("kw", [dict(enforce_eager=True), dict(), dict(max_num_batched_tokens=24, chunked_prefill_tokens=4),
                                dict(max_tokens=5 * dm.PAGE), dict(decode_steps_per_call=4)])
def test_greedy_generation_and_sampling_parameters(kw, tmp_path):
    """The engine's own entry point and scheduler: whole and split prompts, preemption, several steps per call."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = dm.engine(path, "cpu", "float32", **dict(dict(max_tokens=160), **kw))
    prompts = [dm.tokens(n, cfg["vocab"], n) for n in (30, 2, 45, 17, 1)]
    out = [o["token_ids"] for o in llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))]
    for p, o in zip(prompts, out):
        logits = oracle.forward(cfg, w, p + o)[0]
        assert logits[len(p) - 1:-1].argmax(-1).tolist() == o
    if "max_tokens" in kw:
        assert llm.stats.preemptions > 0
    llm.scheduler.block_manager.check_invariants([])
    out = llm.generate(prompts[:2], SamplingParams(temperature=1.0, max_tokens=5, ignore_eos=True))
    assert all(len(o["token_ids"]) == 5 for o in out)


def test_prefixes_that_requests_share(tmp_path):
    """No layer has a state: whole pages of a common prefix are taken from the cache."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = dm.engine(path, "cpu", "float32", max_tokens=160)
    head = dm.tokens(3 * dm.PAGE, cfg["vocab"], 9)
    for tail in (dm.tokens(5, cfg["vocab"], 1), dm.tokens(20, cfg["vocab"], 2)):
        out = llm.generate([head + tail], SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))[0]["token_ids"]
        p = head + tail
        assert oracle.forward(cfg, w, p + out)[0][len(p) - 1:-1].argmax(-1).tolist() == out


def test_layers_that_read_other_rows_keep_none(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    llm = dm.engine(path, "cpu", "float32")
    layout = llm.model_runner.cache_layout
    assert [c.row_width for c in layout] == [24 + 24, 24, 16, 24 + 24]
    assert llm.model_runner.model_type == "darusun" and llm.scheduler.block_manager.prefix_caching


def test_checkpoint_and_config_errors(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)

    def refused(error, match, change_cfg=None, change_w=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        if change_cfg:
            change_cfg(c)
        if change_w:
            change_w(v)
        with pytest.raises(error, match=match):
            dm.engine(dm.save(tmp_path / "bad", c, v), "cpu", "float32")

    for name in ("l0.mlp.e3.up", "l1.mix.sink", "l2.mix.talk", "l3.mix.dq.norm", "l3.mlp.shared.sg", "l0.mlp.router.b", "l1.mlp.act",
                 "final.norm"):
        refused(RuntimeError, name, change_w=lambda v: v.pop(name))
    refused(ValueError, "shape", change_w=lambda v: v.update({"l1.norm1": torch.zeros(39)}))
    refused(ValueError, "shape", change_w=lambda v: v.update({"l0.mix.talk": torch.zeros(3, 3)}))
    refused(ValueError, "shape", change_w=lambda v: v.update({"l1.mlp.act": torch.zeros(3)}))
    refused(ValueError, "other", lambda c: c["layers"][0].update(type="other"))
    refused(ValueError, "other", lambda c: c["layers"][0]["mlp"].update(kind="other"))
    refused(ValueError, "evenly", lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    refused(ValueError, "experts per token", lambda c: c["layers"][3]["mlp"]["router"].update(top=6))
    refused(ValueError, "rotated", lambda c: c["layers"][4]["mixer"]["rot"].update(dims=10))
    refused(ValueError, "rotated", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8))
    refused(ValueError, "kv_from", lambda c: c["layers"][2]["mixer"].update(kv_from=1))
    refused(ValueError, "kv_from", lambda c: c["layers"][2]["mixer"].update(kv_from=3))
    refused(ValueError, "shares", lambda c: c["layers"][2]["mixer"].update(vdim=12))


def test_random_initialisation():
    from fastcache_b200 import LLM
    llm = LLM(dm.config(**MIX), device="cpu", kvcache_block_size=16, num_kvcache_blocks=16, max_model_len=128, max_num_seqs=2)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert len(out[0]["token_ids"]) == 3


def test_trace_run_command(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    toks = dm.tokens(40, cfg["vocab"], 8)
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": toks[30:31], "want": []},
                                     {"id": "q", "tokens": toks[:5], "want": [4]}], "end": ["q"]},
             {"step": 2, "entries": [{"id": "p", "tokens": toks[31:], "want": [8]}], "end": ["p"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([sys.executable, "-m", "fastcache_b200.serving.trace_run", "--model", path, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128", "--device", "cpu"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = oracle.forward(cfg, w, toks)[0]
    got = [torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"])) for i in range(3)]
    for rows, at in zip(got, ([0, 29], [4], [39])):
        assert dm.errors(rows, want[at])[0] < TOL


def test_server(tmp_path):
    from fastcache_b200.serving.server import FastCacheServer
    cfg, w, path = _model(tmp_path, MIX)
    server = FastCacheServer(path, compression_mode="lazy", max_model_len=128, device="cpu", dtype="float32",
                             kvcache_block_size=16, num_kvcache_blocks=32, max_num_seqs=3, tokenizer=False)
    try:
        prompts = [dm.tokens(n, cfg["vocab"], n) for n in (20, 5, 33, 9)]
        futures = [server.submit(p, 6, 0.0) for p in prompts]
        for p, f in zip(prompts, futures):
            out = f.result(60)["token_ids"]
            assert oracle.forward(cfg, w, p + out)[0][len(p) - 1:-1].argmax(-1).tolist() == out
    finally:
        server.shutdown()
