"""Duperax through the engine on CPU (32-bit): cache, state slots, loop passes, streams, scheduler and loader against the plain
statements."""
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import duperax_models as dm
import duperax_oracle as oracle
from fastcache_b200 import SamplingParams
from fastcache_b200.engine.replay import TokenReplay

MIX = dict(layers=[(dm.rglru(width=20, blocks=2, taps=3), dm.dense(24)),
                   (dm.attention(heads=4, kv_heads=2, dim=12, vdim=10, window=18), dm.moe(experts=6, top=2, ff=20)),
                   (dm.rglru(width=18, blocks=3, taps=2), dm.moe(experts=8, top=3, ff=16, groups=2, keep=1)),
                   (dm.chunked(heads=3, kv_heads=1, dim=10, vdim=14, rot=8, chunk=21), None)],
           width=40, vocab=60, loop=(1, 3, 2))
SINGLE = {
    "window": dict(layers=[(dm.attention(), None)]),
    "window of one": dict(layers=[(dm.attention(heads=1, kv_heads=1, dim=8, vdim=8, window=1), None)]),
    "window of a page": dict(layers=[(dm.attention(heads=3, kv_heads=3, dim=9, vdim=16, window=16), dm.dense(9))]),
    "window past the prompt": dict(layers=[(dm.attention(window=500, scale=0.05), None)]),
    "chunks": dict(layers=[(dm.chunked(), None)]),
    "chunks of one": dict(layers=[(dm.chunked(chunk=1), None)]),
    "chunks of a page, all of the head rotated": dict(layers=[(dm.chunked(heads=2, kv_heads=2, dim=12, vdim=7, rot=12, chunk=16), None)]),
    "chunk past the prompt, no scaling, tight cap": dict(layers=[(dm.chunked(chunk=300, scaling=None, softcap=1.0), None)]),
    "scaling by one, ramp of no width": dict(layers=[(dm.chunked(scaling=(1.0, 4096, 1.0, 1.0)), None)]),
    "scaling of every pair": dict(layers=[(dm.chunked(scaling=(4.0, 8, 64.0, 32.0), softcap=50.0), None)]),
    "recurrent unit": dict(layers=[(dm.rglru(), None)]),
    "recurrent unit, one block": dict(layers=[(dm.rglru(width=14, blocks=1, taps=2), None)]),
    "recurrent unit, blocks of one, no memory in the convolution": dict(layers=[(dm.rglru(width=5, blocks=5, taps=1), None)]),
    "recurrent unit, six taps": dict(layers=[(dm.rglru(width=16, blocks=2, taps=6), dm.dense(12, limit=0.3))]),
    "dense": dict(layers=[(dm.rglru(width=8, blocks=1), dm.dense(50))]),
    "dense, wide limit": dict(layers=[(dm.rglru(width=8, blocks=1), dm.dense(17, limit=7.0))]),
    "experts": dict(layers=[(dm.rglru(width=8, blocks=1), dm.moe())]),
    "one group": dict(layers=[(dm.attention(), dm.moe(experts=5, top=3, ff=12, groups=1, keep=1))]),
    "all groups": dict(layers=[(dm.attention(), dm.moe(experts=8, top=2, ff=12, groups=4, keep=4))]),
    "all experts of the kept groups": dict(layers=[(dm.attention(), dm.moe(experts=9, top=6, ff=12, groups=3, keep=2))]),
    "one expert of many": dict(layers=[(dm.attention(), dm.moe(experts=12, top=1, ff=12, groups=4, keep=1))]),
    "one stream": dict(layers=[(dm.attention(), dm.dense(20)), (dm.rglru(), None)], streams=1),
    "five streams": dict(layers=[(dm.attention(), dm.moe()), (dm.rglru(), dm.dense(20))], streams=5),
    "loop from the start": dict(layers=[(dm.attention(window=9), dm.dense(20)), (dm.rglru(), None)], loop=(0, 1, 3)),
    "loop to the end": dict(layers=[(dm.rglru(), None), (dm.chunked(chunk=9), dm.moe())], loop=(1, 2, 2)),
    "loop over everything": dict(layers=[(dm.rglru(), None), (dm.attention(window=9), None)], loop=(0, 2, 2)),
    "loop that runs once": dict(layers=[(dm.rglru(), None), (dm.chunked(), None)], loop=(0, 1, 1), logit_scale=0.5),
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

    def zero(t):
        return 0 * t
    out = {"window": cfg(("layers", 1, "mixer", "mask", "size"), 19), "chunk": cfg(("layers", 3, "mixer", "mask", "size"), 22),
           "softcap": cfg(("layers", 3, "mixer", "softcap"), 14.0), "rotated dimensions": cfg(("layers", 3, "mixer", "rot", "dims"), 6),
           "scaling": lambda c, w: c["layers"][3]["mixer"]["rot"].pop("scaling"), "limit": cfg(("layers", 0, "mlp", "limit"), 1.3),
           "groups": cfg(("layers", 1, "mlp", "router", "groups", "keep"), 3), "top": cfg(("layers", 2, "mlp", "router", "top"), 2),
           "logit scale": cfg(("logit_scale",), 1.4), "passes": cfg(("loop", "times"), 3),
           "correction": tensor("l1.mlp.correction", zero), "gates": swap("l0.mix.ra", "l0.mix.ri"),
           "from and to": tensor("l2.hc1.mix", lambda t: t.T), "connections": swap("l2.hc1.in", "l2.hc2.in"), "out": swap("l0.hc1.out", "l0.hc2.out"),
           "conv": tensor("l0.mix.conv", lambda t: t.flip(1)), "lam": tensor("l2.mix.lam", lambda t: t + 0.3)}
    for name in ("l0.norm2.b", "l1.norm1.b", "final.norm.b", "l3.mix.q.b", "l3.mix.k.b", "l3.mix.v.b", "l0.mix.y.b", "l0.mix.x.b",
                 "l0.mix.conv.b", "l2.mix.ra.b", "l2.mix.ri.b"):
        out[name] = tensor(name, zero)
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


def test_experts_are_weighed_without_the_correction():
    router = dict(experts=6, top=2, groups=dict(count=3, keep=2))
    z, c = torch.tensor([2.0, -1.0, 0.5, 0.4, -3.0, 1.0]), torch.tensor([-3.0, 0.0, -0.1, 0.2, 0.1, -0.6])
    # choice scores: -2.12 .27 | .52 .80 | .15 .13; sums: -1.85, 1.32, .28; the first group is out although expert 1 beats 4
    got = oracle.route(z, c, router)
    assert sorted(got) == [2, 3]
    assert abs(float(sum(got.values())) - 1) < 1e-6 and float(got[2]) > float(got[3])


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
        for name in list(c.state) + (["k_rows", "v_rows"] if c.kv else []):
            getattr(c.module, name).fill_(value)


def test_pages_and_slots_are_used_again(tmp_path):
    """A pool with room for two requests of three pages and two slots, filled with junk first: many requests in turn."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = dm.engine(path, "cpu", "float32", max_tokens=6 * dm.PAGE, requests=2)
    fill_caches(llm, 100.0)
    replay = TokenReplay(llm)
    tables, slots = set(), []
    for k in range(6):
        prompts = {f"x{k}": dm.tokens(35 + k, cfg["vocab"], k), f"y{k}": dm.tokens(20 + k, cfg["vocab"], 50 + k)}
        want = dm.expected(cfg, w, prompts)
        names = list(prompts)
        for n in (names if k % 2 else names[::-1]):
            replay.step([{"id": n, "tokens": prompts[n][:10], "want": []}])
        slots.append(tuple(replay.live[n].state_slot for n in names))
        tables |= {tuple(replay.live[n].block_table) for n in names}
        got = replay.step([{"id": n, "tokens": prompts[n][10:], "want": [len(prompts[n]) - 11]} for n in names], names)
        for i, n in enumerate(names):
            assert dm.errors(got[i:i + 1], want[n][-1:])[0] < TOL
    assert len(set(slots)) > 1 and len(tables) > 2
    llm.scheduler.block_manager.check_invariants([])
    with pytest.raises(RuntimeError, match="slot"):
        for n in "pqr":
            replay.step([{"id": n, "tokens": [1], "want": []}])


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
    spec = dm.attention(heads=4, kv_heads=2, dim=12, vdim=16, window=window)
    for at in (n - 1 - window, n - window, n - 2, 0):
        _pointer(spec, at, n, at >= n - window, tmp_path)


@pytest.mark.parametrize("chunk", [15, 16, 17, 33, 69, 70])
def test_keys_at_the_edges_of_the_chunk(chunk, tmp_path):
    """The same with chunks, which count from the start of the sequence; the last token may be the first of its chunk."""
    n = 70
    spec = dm.chunked(heads=4, kv_heads=2, dim=16, vdim=12, rot=6, chunk=chunk)
    first = (n - 1) // chunk * chunk
    for at in sorted({max(first - 1, 0), min(first, n - 2), n - 2, 0}):
        _pointer(spec, at, n, at >= first, tmp_path)


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


def test_every_pass_keeps_its_own_rows_and_state(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    llm = dm.engine(path, "cpu", "float32")
    layout = llm.model_runner.cache_layout
    assert len(layout) == len(oracle.layer_order(cfg)) == 6 and len({id(c.module) for c in layout}) == 6
    assert [bool(c.kv) for c in layout] == [False, True, False, True, False, True]
    assert llm.model_runner.model_type == "duperax" and llm.config.num_state_slots == 4
    assert not llm.scheduler.block_manager.prefix_caching


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

    for name in ("l1.mlp.e3.up", "l0.hc2.out", "l3.mix.v.b", "l2.mix.ri", "l2.mlp.correction", "final.norm.b"):
        refused(RuntimeError, name, change_w=lambda v: v.pop(name))
    refused(ValueError, "shape", change_w=lambda v: v.update({"l1.norm1": torch.zeros(39)}))
    refused(ValueError, "shape", change_w=lambda v: v.update({"l1.hc1.mix": torch.zeros(2, 2)}))
    refused(ValueError, "other", lambda c: c["layers"][0].update(type="other"))
    refused(ValueError, "other", lambda c: c["layers"][0]["mlp"].update(kind="other"))
    refused(ValueError, "evenly", lambda c: c["layers"][1]["mixer"].update(kv_heads=3))
    refused(ValueError, "equal parts", lambda c: c["layers"][0]["mixer"].update(blocks=3))
    refused(ValueError, "groups", lambda c: c["layers"][1]["mlp"]["router"].update(top=5))
    refused(ValueError, "rotated", lambda c: c["layers"][3]["mixer"]["rot"].update(dims=12))
    refused(ValueError, "loop", lambda c: c["loop"].update(stop=9))


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
