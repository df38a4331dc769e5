"""Bagedra through the engine on CPU (32-bit): cache, state slots, scheduler and loader against the plain statements."""
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import bagedra_models as bm
import bagedra_oracle as oracle
from fastcache_b200 import SamplingParams
from fastcache_b200.engine.replay import TokenReplay

MIX = [bm.gla(heads=2, dim=6, vdim=10), bm.latent(heads=2, dim=12, rot=8, vdim=20, rank=24),
       bm.delta(heads=4, kv_heads=2, dim=8, vdim=12, conv=3), bm.latent(heads=3, dim=10, rot=8, vdim=6, rank=24, kv_from=1)]
SINGLE = {
    "latent": [bm.latent(heads=2, dim=12, rot=8, vdim=20, rank=24)],
    "latent one head": [bm.latent(heads=1, dim=5, rot=2, vdim=3, rank=9)],
    "shared rows": [bm.latent(rank=16, rot=4), bm.latent(heads=1, dim=24, vdim=8, rank=16, rot=4, kv_from=0),
                    bm.latent(heads=5, dim=8, vdim=8, rank=16, rot=4, kv_from=0)],
    "gla": [bm.gla()],
    "gla tau 1, one head": [bm.gla(heads=1, dim=9, vdim=5, tau=1.0)],
    "delta": [bm.delta()],
    "delta no sharing, one tap": [bm.delta(heads=2, kv_heads=2, dim=7, vdim=9, conv=1)],
    "delta two taps": [bm.delta(heads=4, kv_heads=2, dim=8, vdim=8, conv=2)],
    "delta six taps": [bm.delta(heads=2, kv_heads=1, dim=8, vdim=16, conv=6)],
}
TOL = 2e-5


def _model(tmp_path, mixers, seed=0, **kw):
    cfg = bm.config(mixers, **dict(dict(width=40, ff=24, vocab=60), **kw))
    w = bm.weights(cfg, seed=seed, rank=5)
    return cfg, w, bm.save(tmp_path / "m", cfg, w)


def _cuts(n, sizes):
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


@pytest.mark.parametrize("name", list(SINGLE))
@pytest.mark.parametrize("mlp", [True, False])
def test_each_mechanism_whole_and_in_portions(name, mlp, tmp_path):
    cfg, w, path = _model(tmp_path, SINGLE[name], seed=3, no_mlp=() if mlp else (0, 1, 2))
    prompts = {"a": bm.tokens(53, cfg["vocab"], 5)}
    want = bm.expected(cfg, w, prompts)
    llm = bm.engine(path, "cpu", "float32")
    for sizes in ([53], [1], [2], [20, 1, 1, 3], [16, 17, 15]):
        got = bm.feed(llm, prompts, [[("a", n)] for n in _cuts(53, sizes)])
        assert bm.errors(got["a"], want["a"])[0] < TOL, sizes


def test_unequal_requests_together_and_alone(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    prompts = {c: bm.tokens(n, cfg["vocab"], n) for c, n in zip("abcd", (40, 1, 33, 7))}
    want = bm.expected(cfg, w, prompts)
    schedule = [[("a", 3), ("c", 17)], [("b", 1), ("c", 1), ("a", 14)], [("d", 2), ("a", 1)], [("c", 15), ("d", 1)],
                [("a", 20), ("d", 4)]] + [[("a", 1)], [("a", 1)]]
    got = bm.feed(bm.engine(path, "cpu", "float32"), prompts, schedule)
    for i in prompts:
        assert bm.errors(got[i], want[i])[0] < TOL, i


def test_pages_and_slots_are_used_again(tmp_path):
    """A pool with room for two requests of three pages and two slots, filled with junk first: many requests in turn."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = bm.engine(path, "cpu", "float32", max_tokens=6 * bm.PAGE, requests=2)
    for c in llm.model_runner.cache_layout:
        for name in c.state:
            getattr(c.module, name).fill_(100.0)
        if c.row_width:
            c.module.rows.fill_(100.0)
    replay = TokenReplay(llm)
    tables, slots = set(), []
    for k in range(6):
        prompts = {f"x{k}": bm.tokens(35 + k, cfg["vocab"], k), f"y{k}": bm.tokens(20 + k, cfg["vocab"], 50 + k)}
        want = bm.expected(cfg, w, prompts)
        names = list(prompts)
        for n in (names if k % 2 else names[::-1]):
            replay.step([{"id": n, "tokens": prompts[n][:10], "want": []}])
        slots.append(tuple(replay.live[n].state_slot for n in names))
        tables |= {tuple(replay.live[n].block_table) for n in names}
        got = replay.step([{"id": n, "tokens": prompts[n][10:], "want": [len(prompts[n]) - 11]} for n in names], names)
        for i, n in enumerate(names):
            assert bm.errors(got[i:i + 1], want[n][-1:])[0] < TOL
    assert len(set(slots)) > 1 and len(tables) > 2
    llm.scheduler.block_manager.check_invariants([])
    with pytest.raises(RuntimeError, match="slot"):
        for n in "pqr":
            replay.step([{"id": n, "tokens": [1], "want": []}])


@pytest.mark.parametrize("at", [0, 1, 15, 16, 17, 31, 32, 47])
def test_a_single_far_key(at, tmp_path):
    n = 70
    cfg, w, prompt = bm.pointer_model(at, n, bm.latent(heads=2, dim=12, rot=8, vdim=20, rank=24))
    without = list(prompt)
    without[at] = 5
    want = oracle.forward(cfg, w, prompt)[0]
    assert bm.errors(oracle.forward(cfg, w, without)[0][-1:], want[-1:])[0] > 0.2
    llm = bm.engine(bm.save(tmp_path / "m", cfg, w), "cpu", "float32")
    for cut in ([n], [n - 1, 1], [at + 1, n - at - 2, 1], [32, 31, n - 63]):
        got = bm.feed(llm, {"a": prompt}, [[("a", c)] for c in cut if c])
        assert bm.errors(got["a"], want)[0] < TOL, cut


def test_long_decoding(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    prompts = {"a": bm.tokens(150, cfg["vocab"], 1), "b": bm.tokens(140, cfg["vocab"], 2)}
    got = bm.feed(bm.engine(path, "cpu", "float32"), prompts, [[("a", 12), ("b", 2)]] + [[("a", 1), ("b", 1)]] * 138)
    want = bm.expected(cfg, w, prompts)
    assert all(bm.errors(got[i], want[i])[0] < TOL for i in prompts)


@pytest.mark.parametrize("kw", [dict(enforce_eager=True), dict(), dict(max_num_batched_tokens=24, chunked_prefill_tokens=4),
                                dict(max_tokens=5 * bm.PAGE), dict(decode_steps_per_call=4)])
def test_greedy_generation_and_sampling_parameters(kw, tmp_path):
    """The engine's own entry point and scheduler: whole and split prompts, preemption, several steps per call."""
    cfg, w, path = _model(tmp_path, MIX)
    llm = bm.engine(path, "cpu", "float32", **dict(dict(max_tokens=160), **kw))
    prompts = [bm.tokens(n, cfg["vocab"], n) for n in (30, 2, 45, 17, 1)]
    out = [o["token_ids"] for o in llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))]
    for p, o in zip(prompts, out):
        logits = oracle.forward(cfg, w, p + o)[0]
        assert logits[len(p) - 1:-1].argmax(-1).tolist() == o
    if "max_tokens" in kw:
        assert llm.stats.preemptions > 0
    llm.scheduler.block_manager.check_invariants([])
    out = llm.generate(prompts[:2], SamplingParams(temperature=1.0, max_tokens=5, ignore_eos=True))
    assert all(len(o["token_ids"]) == 5 for o in out)


def test_abort_and_recovery_give_slots_back(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    llm = bm.engine(path, "cpu", "float32")
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    a, b = (llm.add_request(bm.tokens(20, cfg["vocab"], s), sp) for s in (1, 2))
    llm.step()
    llm.step()
    assert llm.abort_request(a.seq_id) and llm.recover() == 1
    while not llm.is_finished():
        llm.step()
    logits = oracle.forward(cfg, w, b.token_ids)[0]
    assert logits[19:-1].argmax(-1).tolist() == b.completion_token_ids
    llm.scheduler.block_manager.check_invariants([])


def test_settings_that_do_not_apply(tmp_path, capsys):
    cfg, w, path = _model(tmp_path, MIX)
    llm = bm.engine(path, "cpu", "float32", prefix_caching=True, enable_compression=True, compression_backend="kvpress",
                    kvpress_method="knorm")
    assert "compression disabled" in capsys.readouterr().out
    assert not llm.enable_compression and not llm.scheduler.block_manager.prefix_caching
    assert llm.model_runner.model_type == "bagedra" and llm.config.num_state_slots == 4


def test_checkpoint_errors(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    short = dict(w)
    short.pop("l2.mix.k.conv")
    with pytest.raises(RuntimeError, match="l2.mix.k.conv"):
        bm.engine(bm.save(tmp_path / "short", cfg, short), "cpu", "float32")
    bad = json.loads(json.dumps(cfg))
    bad["layers"][3]["mixer"]["kv_from"] = 0
    with pytest.raises(ValueError, match="kv_from"):
        bm.engine(bm.save(tmp_path / "bad", bad, w), "cpu", "float32")
    bad["layers"][3]["type"] = "other"
    with pytest.raises(ValueError, match="other"):
        bm.engine(bm.save(tmp_path / "bad2", bad, w), "cpu", "float32")


def test_random_initialisation():
    from fastcache_b200 import LLM
    cfg = bm.config(MIX, width=40, ff=24, vocab=60)
    llm = LLM(cfg, device="cpu", kvcache_block_size=16, num_kvcache_blocks=16, max_model_len=128, max_num_seqs=2)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert len(out[0]["token_ids"]) == 3


def test_trace_run_command(tmp_path):
    cfg, w, path = _model(tmp_path, MIX)
    toks = bm.tokens(40, cfg["vocab"], 8)
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
        assert bm.errors(rows, want[at])[0] < TOL


@pytest.mark.parametrize("mode", ["lazy", "none"])
def test_server_with_its_default_settings(mode, tmp_path):
    from fastcache_b200.serving.server import FastCacheServer
    cfg, w, path = _model(tmp_path, MIX)
    server = FastCacheServer(path, compression_mode=mode, max_model_len=128, device="cpu", dtype="float32",
                             kvcache_block_size=16, num_kvcache_blocks=32, max_num_seqs=3, tokenizer=False)
    try:
        prompts = [bm.tokens(n, cfg["vocab"], n) for n in (20, 5, 33, 9)]
        futures = [server.submit(p, 6, 0.0) for p in prompts]
        for p, f in zip(prompts, futures):
            out = f.result(60)["token_ids"]
            assert oracle.forward(cfg, w, p + out)[0][len(p) - 1:-1].argmax(-1).tolist() == out
    finally:
        server.shutdown()
