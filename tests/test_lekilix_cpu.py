"""Lekilix through the engine on CPU (32-bit): cache, state slots, loop passes, scheduler and loader against the plain
statements."""
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import lekilix_models as lm
import lekilix_oracle as oracle
from fastcache_b200 import SamplingParams
from fastcache_b200.engine.replay import TokenReplay

MIX = dict(layers=[(lm.mlstm(heads=2, dim=6, vdim=10), lm.dense(24)),
                   (lm.attention(heads=4, kv_heads=2, dim=12, rot=6, window=18), lm.moe(experts=6, top=2, ff=20)),
                   (lm.mlstm(heads=3, dim=8, vdim=6, cap=5.0), lm.moe(experts=4, top=3, ff=16, limit=1.0)),
                   (lm.attention(heads=3, kv_heads=1, dim=10, rot=10, window=33), None)],
           width=40, vocab=60, loop=(1, 3, 2))
SINGLE = {
    "attention": dict(layers=[(lm.attention(), None)]),
    "attention, own key heads, all of the head rotated": dict(layers=[(lm.attention(heads=3, kv_heads=3, dim=10, rot=10, window=7), None)]),
    "attention, one head, window of one": dict(layers=[(lm.attention(heads=1, kv_heads=1, dim=8, rot=2, window=1), None)]),
    "attention, window of a page": dict(layers=[(lm.attention(window=16, base=100.0), lm.dense(9))]),
    "attention, window past the prompt": dict(layers=[(lm.attention(window=500, scale=0.05), None)]),
    "mlstm": dict(layers=[(lm.mlstm(), None)]),
    "mlstm, one head, tight cap": dict(layers=[(lm.mlstm(heads=1, dim=7, vdim=5, cap=1.0), None)]),
    "mlstm, wide cap": dict(layers=[(lm.mlstm(heads=2, dim=8, vdim=16, cap=30.0), None)]),
    "dense": dict(layers=[(lm.mlstm(heads=1, dim=4, vdim=4), lm.dense(50))]),
    "experts": dict(layers=[(lm.mlstm(heads=1, dim=4, vdim=4), lm.moe())]),
    "one expert of many": dict(layers=[(lm.attention(), lm.moe(experts=9, top=1, ff=12, limit=0.5))]),
    "all experts": dict(layers=[(lm.attention(), lm.moe(experts=3, top=3, ff=12, limit=7.0))]),
    "one expert": dict(layers=[(lm.attention(), lm.moe(experts=1, top=1, ff=12))]),
    "loop from the start": dict(layers=[(lm.attention(window=9), lm.dense(20)), (lm.mlstm(), None)], loop=(0, 1, 3)),
    "loop to the end": dict(layers=[(lm.mlstm(), None), (lm.attention(window=9), lm.moe())], loop=(1, 2, 2)),
    "loop over everything": dict(layers=[(lm.mlstm(), None), (lm.attention(window=9), None)], loop=(0, 2, 2)),
    "loop that runs once": dict(layers=[(lm.mlstm(), None), (lm.attention(window=9), None)], loop=(0, 1, 1)),
}
TOL = 2e-5


def _model(tmp_path, spec, seed=0, **kw):
    cfg = lm.config(**dict(spec, **kw))
    w = lm.weights(cfg, seed=seed)
    return cfg, w, lm.save(tmp_path / "m", cfg, w)


def _cuts(n, sizes):
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


@pytest.mark.parametrize("name", list(SINGLE))
def test_each_mechanism_whole_and_in_portions(name, tmp_path):
    cfg, w, path = _model(tmp_path, SINGLE[name], seed=3)
    prompts = {"a": lm.tokens(53, cfg["vocab"], 5)}
    want = lm.expected(cfg, w, prompts)
    llm = lm.engine(path, "cpu", "float32")
    for sizes in ([53], [1], [2], [20, 1, 1, 3], [16, 17, 15]):
        got = lm.feed(llm, prompts, [[("a", n)] for n in _cuts(53, sizes)])
        assert lm.errors(got["a"], want["a"])[0] < TOL, sizes


@pytest.mark.parametrize("change", ["sink", "window", "rotation", "cap", "limit", "table", "x0", "norm", "first token"])
def test_the_random_models_show_a_fault(change):
    """Every mechanism of the models above leaves a trace in the logits: change it in the plain statements and look."""
    cfg = lm.config(**MIX)
    w = lm.weights(cfg)
    prompt = lm.tokens(50, cfg["vocab"], 1)
    want = oracle.forward(cfg, w, prompt)[0]
    c, v = json.loads(json.dumps(cfg)), dict(w)
    att, mem = c["layers"][1], c["layers"][2]
    if change == "sink":
        v["l1.mix.sink"] = torch.full_like(v["l1.mix.sink"], -30.0)
    elif change == "window":
        att["mixer"]["mask"]["size"] += 1
    elif change == "rotation":
        att["mixer"]["rot"]["dims"] -= 2
    elif change == "cap":
        mem["mixer"]["gate_cap"] += 1.0
    elif change == "limit":
        att["mlp"]["expert"]["limit"] += 0.2
    elif change == "table":
        v["l1.mlp.table"] = v["l1.mlp.table"].roll(1, 0)
    elif change == "x0":
        v["loop.in"] = v["loop.in"].clone()
        v["loop.in"][:, cfg["width"]:] = 0
    elif change == "norm":
        v["l2.norm1"] = v["l2.norm1"] + 0.1
    else:
        prompt = [(prompt[0] + 1) % cfg["vocab"]] + prompt[1:]
    assert lm.errors(oracle.forward(c, v, prompt)[0][-20:], want[-20:])[0] > 100 * TOL


def test_unequal_requests_together_and_alone(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    prompts = {c: lm.tokens(n, cfg["vocab"], n) for c, n in zip("abcd", (40, 1, 33, 7))}
    want = lm.expected(cfg, w, prompts)
    schedule = [[("a", 3), ("c", 17)], [("b", 1), ("c", 1), ("a", 14)], [("d", 2), ("a", 1)], [("c", 15), ("d", 1)],
                [("a", 20), ("d", 4)]] + [[("a", 1)], [("a", 1)]]
    got = lm.feed(lm.engine(path, "cpu", "float32"), prompts, schedule)
    for i in prompts:
        assert lm.errors(got[i], want[i])[0] < TOL, i


def fill_caches(llm, value):
    for c in llm.model_runner.cache_layout:
        for name in list(c.state) + (["k_rows", "v_rows"] if c.kv else []):
            getattr(c.module, name).fill_(value)


def test_pages_and_slots_are_used_again(tmp_path):
    """A pool with room for two requests of three pages and two slots, filled with junk first: many requests in turn."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = lm.engine(path, "cpu", "float32", max_tokens=6 * lm.PAGE, requests=2)
    fill_caches(llm, 100.0)
    replay = TokenReplay(llm)
    tables, slots = set(), []
    for k in range(6):
        prompts = {f"x{k}": lm.tokens(35 + k, cfg["vocab"], k), f"y{k}": lm.tokens(20 + k, cfg["vocab"], 50 + k)}
        want = lm.expected(cfg, w, prompts)
        names = list(prompts)
        for n in (names if k % 2 else names[::-1]):
            replay.step([{"id": n, "tokens": prompts[n][:10], "want": []}])
        slots.append(tuple(replay.live[n].state_slot for n in names))
        tables |= {tuple(replay.live[n].block_table) for n in names}
        got = replay.step([{"id": n, "tokens": prompts[n][10:], "want": [len(prompts[n]) - 11]} for n in names], names)
        for i, n in enumerate(names):
            assert lm.errors(got[i:i + 1], want[n][-1:])[0] < TOL
    assert len(set(slots)) > 1 and len(tables) > 2
    llm.scheduler.block_manager.check_invariants([])
    with pytest.raises(RuntimeError, match="slot"):
        for n in "pqr":
            replay.step([{"id": n, "tokens": [1], "want": []}])


@pytest.mark.parametrize("window", [15, 16, 17, 32, 40])
def test_keys_at_the_edges_of_the_window(window, tmp_path):
    """One key carries the whole answer: just inside the window it decides the last logits, just outside it is not there."""
    n = 70
    spec = lm.attention(heads=4, kv_heads=2, dim=12, rot=6, window=window)
    for at in (n - 1 - window, n - window, n - 2, 0):
        cfg, w, prompt = lm.pointer_model(spec, at, n)
        want = oracle.forward(cfg, w, prompt)[0]
        without = list(prompt)
        without[at] = 5
        seen = lm.errors(oracle.forward(cfg, w, without)[0][-1:], want[-1:])[0]
        assert seen > 0.5 if at >= n - window else seen < 1e-6
        llm = lm.engine(lm.save(tmp_path / f"m{at}", cfg, w), "cpu", "float32")
        for cut in ([n], [n - 1, 1], [at + 1, n - at - 2, 1], [32, 31, n - 63]):
            got = lm.feed(llm, {"a": prompt}, [[("a", c)] for c in cut if c])
            assert lm.errors(got["a"], want)[0] < TOL, (at, cut)


def test_long_decoding(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    prompts = {"a": lm.tokens(150, cfg["vocab"], 1), "b": lm.tokens(140, cfg["vocab"], 2)}
    got = lm.feed(lm.engine(path, "cpu", "float32"), prompts, [[("a", 12), ("b", 2)]] + [[("a", 1), ("b", 1)]] * 138)
    want = lm.expected(cfg, w, prompts)
    assert all(lm.errors(got[i], want[i])[0] < TOL for i in prompts)


@pytest.mark.parametrize("kw", [dict(enforce_eager=True), dict(), dict(max_num_batched_tokens=24, chunked_prefill_tokens=4),
                                dict(max_tokens=5 * lm.PAGE), dict(decode_steps_per_call=4)])
def test_greedy_generation_and_sampling_parameters(kw, tmp_path):
    """The engine's own entry point and scheduler: whole and split prompts, preemption, several steps per call."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = lm.engine(path, "cpu", "float32", **dict(dict(max_tokens=160), **kw))
    prompts = [lm.tokens(n, cfg["vocab"], n) for n in (30, 2, 45, 17, 1)]
    out = [o["token_ids"] for o in llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))]
    for p, o in zip(prompts, out):
        logits = oracle.forward(cfg, w, p + o)[0]
        assert logits[len(p) - 1:-1].argmax(-1).tolist() == o
    if "max_tokens" in kw:
        assert llm.stats.preemptions > 0
    llm.scheduler.block_manager.check_invariants([])
    out = llm.generate(prompts[:2], SamplingParams(temperature=1.0, max_tokens=5, ignore_eos=True))
    assert all(len(o["token_ids"]) == 5 for o in out)


def test_attention_only_model_needs_no_slots(tmp_path):
    cfg, w, path = _model(tmp_path, SINGLE["attention"])
    llm = lm.engine(path, "cpu", "float32")
    out = llm.generate([[1, 2, 3], [4]], SamplingParams(temperature=0.0, max_tokens=30, ignore_eos=True))
    for p, o in zip(([1, 2, 3], [4]), out):
        logits = oracle.forward(cfg, w, p + o["token_ids"])[0]
        assert logits[len(p) - 1:-1].argmax(-1).tolist() == o["token_ids"]


def test_every_pass_keeps_its_own_rows_and_state(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    llm = lm.engine(path, "cpu", "float32")
    layout = llm.model_runner.cache_layout
    assert len(layout) == len(oracle.layer_order(cfg)) == 6 and len({id(c.module) for c in layout}) == 6
    assert [bool(c.kv) for c in layout] == [False, True, False, True, False, True]
    assert llm.model_runner.model_type == "lekilix" and llm.config.num_state_slots == 4
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
            lm.engine(lm.save(tmp_path / "bad", c, v), "cpu", "float32")

    refused(RuntimeError, "l1.mlp.e3.up", change_w=lambda v: v.pop("l1.mlp.e3.up"))
    refused(RuntimeError, "loop.in", change_w=lambda v: v.pop("loop.in"))
    refused(ValueError, "shape", change_w=lambda v: v.update({"l1.norm1": torch.zeros(39)}))
    refused(ValueError, "experts outside", change_w=lambda v: v.update({"l1.mlp.table": v["l1.mlp.table"] + 1}))
    refused(ValueError, "other", lambda c: c["layers"][0].update(type="other"))
    refused(ValueError, "other", lambda c: c["layers"][0]["mlp"].update(kind="other"))
    refused(ValueError, "values", lambda c: c["layers"][1]["mixer"].update(vdim=8))
    refused(ValueError, "evenly", lambda c: c["layers"][1]["mixer"].update(kv_heads=3))
    refused(ValueError, "loop", lambda c: c["loop"].update(stop=9))


def test_random_initialisation():
    from fastcache_b200 import LLM
    llm = LLM(lm.config(**MIX), device="cpu", kvcache_block_size=16, num_kvcache_blocks=16, max_model_len=128, max_num_seqs=2)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert len(out[0]["token_ids"]) == 3


def test_trace_run_command(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    toks = lm.tokens(40, cfg["vocab"], 8)
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
        assert lm.errors(rows, want[at])[0] < TOL


def test_server(tmp_path):
    from fastcache_b200.serving.server import FastCacheServer
    cfg, w, path = _model(tmp_path, MIX)
    server = FastCacheServer(path, compression_mode="lazy", max_model_len=128, device="cpu", dtype="float32",
                             kvcache_block_size=16, num_kvcache_blocks=32, max_num_seqs=3, tokenizer=False)
    try:
        prompts = [lm.tokens(n, cfg["vocab"], n) for n in (20, 5, 33, 9)]
        futures = [server.submit(p, 6, 0.0) for p in prompts]
        for p, f in zip(prompts, futures):
            out = f.result(60)["token_ids"]
            assert oracle.forward(cfg, w, p + out)[0][len(p) - 1:-1].argmax(-1).tolist() == out
    finally:
        server.shutdown()
