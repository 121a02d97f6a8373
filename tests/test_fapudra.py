"""The Fapudra family through the engine (block pool, scheduler, sampler, trace replay) against the plain equations of
fapudra_oracle: whole prompts, single tokens, portions, mixed batches, reused blocks, generation."""
import copy
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import fapudra_helpers as hlp
import fapudra_oracle as oracle
from decoder_helpers import LIMIT, PLACES, check, greedy, greedy_within_rounding, run_batch
from fapudra_helpers import CONFIGS
from ksanallm_b200.config import EngineConfig, MlpSpec, MoeSpec, ParallelSpec, StateSpaceSpec, model_config_from_hf
from ksanallm_b200.llm import LLM
from ksanallm_b200.models.weights import DictSource, build_model
from ksanallm_b200.ops import native

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
NAMES = sorted(CONFIGS)


@functools.lru_cache(maxsize=None)
def weights_of(name):
    return hlp.of(name)


@functools.lru_cache(maxsize=None)
def truth(name, n, seed=0):
    """(tokens, logits of every position) of a seeded request."""
    t = hlp.tokens(CONFIGS[name], n, seed)
    return t, oracle.forward(t, CONFIGS[name], weights_of(name))


def engine(name, device, dtype, **kw):
    return hlp.engine(CONFIGS[name], weights_of(name), device, dtype, **kw)


# ------------------------------------------------------------------------------------------------ one request
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_portions_and_single_tokens(name, device, dtype):
    t, want = truth(name, 150)
    eng = engine(name, device, dtype)
    for sizes in ([150], [2], [40, 1, 2, 17, 3, 1, 1, 30], [15, 2, 47, 3], [100, 1], [16]):
        check(hlp.run_portions(eng, t, sizes), want, dtype, device)
    short = 150 if device == "cuda" else 50
    check(hlp.run_portions(eng, t[:short], [1]), want[:short], dtype, device)
    for n in (1, 2, 16, 17):
        check(hlp.run_portions(eng, t[:n], [n]), want[:n], dtype, device)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("name", ["unequal", "odd", "wide"])
def test_stream_after_every_layer(name, device, dtype):
    t, streams = hlp.tokens(CONFIGS[name], 60, 3), []
    oracle.forward(t, CONFIGS[name], weights_of(name), streams)
    eng = engine(name, device, dtype)
    got = []
    eng.model.stream_hook = lambda r, x: got.append(x[:, :CONFIGS[name]["width"]].float().cpu().clone())
    hlp.run_portions(eng, t, [60])
    assert len(got) == len(streams) == len(CONFIGS[name]["layers"])
    for a, b in zip(got, streams):
        assert float((a - b).abs().max() / b.abs().max()) < (1e-5 if dtype == torch.float32 else 5e-2)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("name", ["long", "unequal"])
def test_long_decoding(name, device, dtype):
    n = 400 if device == "cuda" else 100
    t, want = truth(name, n, 7)
    eng = engine(name, device, dtype)
    check(hlp.run_portions(eng, t, [3] + [1] * n), want, dtype, device)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("block_tokens", [8, 32, 5])
def test_other_block_sizes(block_tokens, device, dtype):
    t, want = truth("unequal", 150)
    eng = engine("unequal", device, dtype, block_tokens=block_tokens, max_len=150)
    check(hlp.run_portions(eng, t, [33, 1, 1, 50, 2]), want, dtype, device)


# ------------------------------------------------------------------------------------------------ batches
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_and_reused_blocks_and_slots(name, device, dtype):
    lens = (150, 33, 1, 97, 64, 17, 128, 5)
    cases = [truth(name, n, k) for k, n in enumerate(lens)]
    # room for four live requests at a time, far less than for all eight: blocks are handed out again
    eng = engine(name, device, dtype, blocks=31, max_len=160, max_batch_size=4)
    for seed in (0, 1) if device == "cuda" else (0,):
        for got, (_, want) in zip(run_batch(eng, [t for t, _ in cases], seed), cases):
            check(got, want, dtype, device)
    st = eng.scheduler.stats()
    assert st["used_blocks"] == 0 and eng.scheduler.check_invariants()[0]


# ------------------------------------------------------------------------------------------------ generation
def assert_greedy(name, prompt, out, dtype):
    greedy_within_rounding(oracle.forward(prompt + out[:-1], CONFIGS[name], weights_of(name))[len(prompt) - 1:], out, dtype)


PROMPTS = (70, 1, 33, 18, 96, 2)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("options", [{}, {"split_fuse_token_num": 24}, {"enable_auto_prefix_cache": True, "split_fuse_token_num": 40},
                                     {"graphs": True}, {"max_step_tokens": 32}], ids=["plain", "split", "prefix", "graphs", "chunks"])
def test_greedy_generation(options, device, dtype):
    if options.get("graphs") and device == "cpu":
        pytest.skip("CUDA graphs")
    for name in ("unequal", "odd"):
        eng = engine(name, device, dtype, blocks=80, max_len=200, **options)
        prompts = [hlp.tokens(CONFIGS[name], n, 20 + k) for k, n in enumerate(PROMPTS)]
        for again in range(2):                              # the second time blocks and slots are used again
            reqs = eng.generate(prompts, greedy(16))
            for p, r in zip(prompts, reqs):
                assert r.status_code == 0 and len(r.outputs[0].tokens) == 16
                if again or len(p) < 40:
                    assert_greedy(name, p, r.outputs[0].tokens, dtype)
        if options.get("enable_auto_prefix_cache"):         # states cannot be shared: nothing is
            assert eng.scheduler.stats()["prefix_hit_tokens"] == 0
        if options.get("graphs"):
            assert eng.runner.graph_replays > 10
            eng.runner.release_graphs()
    if device == "cuda":
        native.check_err_flag("cuda")


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("mode,host", [(0, 64), (1, 0)], ids=["swap", "recompute"])
def test_generation_under_memory_pressure(mode, host, device, dtype):
    name = "unequal"
    eng = engine(name, device, dtype, blocks=22, max_len=120, host_blocks=host, preempt_mode=mode)
    prompts = [hlp.tokens(CONFIGS[name], n, 40 + n) for n in (50, 47, 40, 45)]
    for p, r in zip(prompts, eng.generate(prompts, greedy(50))):
        assert r.status_code == 0 and len(r.outputs[0].tokens) == 50
        assert_greedy(name, p, r.outputs[0].tokens, dtype)
    st = eng.scheduler.stats()
    assert (st["preempt_swap"] if mode == 0 else st["preempt_recompute"]) > 0
    assert eng.scheduler.check_invariants()[0]


@pytest.mark.parametrize("device,dtype", PLACES)
def test_forked_siblings_and_beams(device, dtype):
    name, n = "unequal", 37
    p = hlp.tokens(CONFIGS[name], n, 50)
    eng = engine(name, device, dtype, blocks=80, max_len=200)
    s = greedy(20)
    s.num_return_sequences = 3
    (r,) = eng.generate([p], s)
    for o in r.outputs:
        assert_greedy(name, p, o.tokens, dtype)
    s = greedy(12)
    s.num_beams = 3
    (r,) = eng.generate([p], s)
    assert r.status_code == 0 and all(len(o.tokens) == 12 for o in r.outputs)

    def score(out):
        rows = oracle.forward(p + out[:-1], CONFIGS[name], weights_of(name))[n - 1:]
        return sum(float(torch.log_softmax(row, -1)[t]) for row, t in zip(rows, out))

    (g,) = eng.generate([p], greedy(12))
    assert max(score(o.tokens) for o in r.outputs) >= score(g.outputs[0].tokens) - 0.5


@pytest.mark.parametrize("device,dtype", PLACES)
def test_forward_targets_and_spliced_embeddings(device, dtype):
    """Hidden states, per-position logits and replaced embedding rows of the /forward interface."""
    name, c = "odd", CONFIGS["odd"]                         # width 70: rows are padded inside
    t, want = truth(name, 150)
    eng = engine(name, device, dtype)
    r = eng.add_request(t[:30], greedy(1), request_target={
        "transformer": {"slice_pos": [[3, 5]], "token_reduce_mode": "GATHER_ALL"},
        "logits": {"slice_pos": [[0, 20]], "token_reduce_mode": "GATHER_TOKEN_ID"}})
    while not r.done.is_set():
        eng.step()
    streams = []
    oracle.forward(t[:30], c, weights_of(name), streams)
    got = r.response["transformer"]
    assert got.shape == (3, 70)
    tol = 1e-4 if dtype == torch.float32 else 0.1
    assert float((got - streams[-1][3:6]).abs().max() / streams[-1].abs().max()) < tol
    probs = torch.softmax(want[:21], -1)[torch.arange(21), torch.tensor(t[1:22])]
    assert torch.allclose(r.response["logits"].reshape(-1), probs, atol=tol)
    emb = torch.randn(1, 70, generator=torch.Generator().manual_seed(4)).bfloat16().float() * 2
    q = eng.add_request(t[:10], greedy(1), refit=([9], [emb]))
    while not q.done.is_set():
        eng.step()
    rows = oracle.forward(t[:10], c, weights_of(name), splice={9: emb[0]})
    greedy_within_rounding(rows[9:], q.outputs[0].tokens, dtype)


# ------------------------------------------------------------------------------------------------ from a checkpoint
@pytest.mark.parametrize("device,dtype", PLACES)
def test_served_from_a_checkpoint(tmp_path, device, dtype):
    name = "long"
    hlp.save_checkpoint(str(tmp_path), CONFIGS[name], weights_of(name))
    ec = EngineConfig()
    ec.model_dir = str(tmp_path)
    ec.batch_scheduler.max_token_len = 128
    ec.block_manager.device_blocks_num = 40
    ec.block_manager.host_blocks_num = 4
    llm = LLM(ec, device=device, dtype=dtype)
    prompts = [hlp.tokens(CONFIGS[name], n, 60 + n) for n in (20, 3)]
    for p, r in zip(prompts, llm.generate(prompts, greedy(16))):
        assert_greedy(name, p, r.outputs[0].tokens, dtype)
    llm.shutdown()


@pytest.mark.parametrize("device,dtype", PLACES)
def test_trace_replay_command(tmp_path, device, dtype):
    name = "unequal"
    model, out = tmp_path / "model", tmp_path / "out"
    out.mkdir()
    hlp.save_checkpoint(str(model), CONFIGS[name], weights_of(name))
    (ta, wa), (tb, wb) = truth(name, 150, 0), truth(name, 64, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:21], "want": [0, 20]}, {"id": "b", "tokens": tb[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[1:2], "want": [0]}, {"id": "a", "tokens": ta[21:60], "want": [38, 2]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": tb[2:64], "want": []}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": ta[:128], "want": [127]}], "end": ["a"]}]
    kind = {torch.float32: "float32", torch.bfloat16: "bfloat16"}[dtype]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", kind, "--out", str(out),
                        "--max-tokens", "128", "--device", device], input="".join(json.dumps(s) + "\n" for s in steps),
                       text=True, capture_output=True, timeout=600, cwd=str(tmp_path))
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    got = {i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, 203) for i in (0, 1, 3)}
    assert sorted(os.listdir(out)) == ["0.f32", "1.f32", "3.f32"]
    for i, want in ((0, wa[[0, 20]]), (1, torch.stack([wb[1], wa[59], wa[23]])), (3, wa[[127]])):
        check(got[i], want, dtype, "cpu")


# ------------------------------------------------------------------------------------------------ configuration, loading
def test_configuration_is_read():
    c = model_config_from_hf(copy.deepcopy(CONFIGS["unequal"]))
    assert (c.model_type, c.hidden_size, c.vocab_size, c.num_layers, c.max_token_len) == ("fapudra", 72, 203, 4, 512)
    assert (c.logit_softcap, c.emb_scale, c.rms_norm_eps, c.tie_word_embeddings) == (24.0, 3.0, 1e-5, False)
    a, b = c.layer_specs[0].mixer, c.layer_specs[1].mixer
    assert isinstance(a, StateSpaceSpec) and (a.heads, a.vdim, a.state, a.groups, a.taps, a.norm_groups) == (6, 16, 24, 2, 3, 3)
    assert isinstance(b, ParallelSpec) and (b.attention_scale, b.recurrence_scale) == (1.25, 0.8)
    left, right = b.attention, b.recurrence
    assert (left.heads, left.kv_heads, left.dim, left.window, left.keep_first, left.bias_far, left.sigmoid) == (6, 2, 24, 20, 5, 40, True)
    assert (right.heads, right.kv_heads, right.dim, right.vdim, right.taps) == (4, 2, 16, 24, 4)
    e = c.layer_specs[0].mlp
    assert isinstance(e, MoeSpec) and (e.router.experts, e.router.top, e.router.groups, e.router.keep_groups) == (15, 4, 5, 3)
    assert (e.router.scoring, e.router.renorm, e.router.group_top) == ("softmax", True, 1)
    assert isinstance(e.expert, MlpSpec) and (e.expert.size, e.expert.limit, e.expert.alpha, e.expert.offset) == (24, 1.3, 1.702, 1.0)
    assert c.layer_specs[1].mlp is None
    p = model_config_from_hf(copy.deepcopy(CONFIGS["plain"])).layer_specs[0].mixer.attention
    assert (p.window, p.keep_first) == (0, 0)


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][0].update(type="convolution"), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c["layers"][0]["mixer"].update(groups=4), lambda c: c["layers"][0]["mixer"].update(norm_groups=7),
    lambda c: c["layers"][0]["mixer"].update(conv=0), lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4),
    lambda c: c["layers"][1]["mixer"]["left"].update(vdim=16), lambda c: c["layers"][1]["mixer"]["left"].update(bias_max=0),
    lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), lambda c: c["layers"][1]["mixer"]["right"].update(kv_heads=3),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), lambda c: c["layers"][0]["mlp"]["router"].update(top=10),
    lambda c: c.update(max_positions=0), lambda c: c.update(layers=[])])
def test_unknown_configurations_are_refused(edit):
    c = copy.deepcopy(CONFIGS["unequal"])
    edit(c)
    with pytest.raises(ValueError):
        model_config_from_hf(c)


def test_wrong_shapes_and_unsupported_options_are_refused():
    name = "unequal"
    for key in ("l0.mix.in", "l0.mlp.e3.down", "l1.mix.right.a2", "l1.mix.left.pb", "pos"):
        w = dict(weights_of(name))
        w[key] = w[key][:-1]
        with pytest.raises(ValueError, match=key):
            hlp.build(CONFIGS[name], w, "cpu", torch.float32)
    m = hlp.build(CONFIGS[name], weights_of(name), "cpu", torch.float32)
    assert m.weight_bytes() > 0 and m.state_bytes() % 16 == 0
    with pytest.raises(ValueError):
        m.allocate_kv_cache(4, 16, torch.float8_e4m3fn)
    with pytest.raises(ValueError):
        engine(name, "cpu", torch.float32, enable_auto_prefix_cache=True, min_flexible_cache_num=16)
    cfg = model_config_from_hf(copy.deepcopy(CONFIGS["odd"]))
    with pytest.raises(ValueError):
        build_model(cfg, DictSource(weights_of("odd"), "fapudra"), 0, 3)
    with pytest.raises(ValueError):
        build_model(cfg, DictSource(weights_of("odd"), "fapudra"), layer_range=(0, 0))


def test_positions_end_with_the_table():
    c = copy.deepcopy(CONFIGS["plain"])
    c["max_positions"] = 48
    w = dict(weights_of("plain"))
    w["pos"] = w["pos"][:48]
    eng = hlp.engine(c, w, "cpu", torch.float32, blocks=16)
    assert eng.sched_cfg.max_token_len == 48
    t = hlp.tokens(c, 40)
    (r,) = eng.generate([t], greedy(20))
    assert r.status_code == 0 and len(r.outputs[0].tokens) == 8
    assert eng.add_request(t + t, greedy(1)).status_code != 0


def test_checked_steps(monkeypatch):
    """The engine's own bounds checks cover the state slots."""
    from ksanallm_b200.ops import checks
    monkeypatch.setenv("KSANA_CHECK_INPUTS", "1")
    eng = engine("plain", "cpu", torch.float32, max_batch_size=2)
    t, want = truth("plain", 150)
    check(hlp.run_portions(eng, t[:40], [9, 1, 30]), want[:40], torch.float32, "cpu")
    seen = []
    monkeypatch.setattr(checks, "check_step", lambda step, model: seen.append(step))
    a, b = eng.open_given(), eng.open_given()
    eng.step_given([(a, t[:5], []), (b, t[:3], [])])
    args = (eng.model.kv_cache.shape[0], eng.model.block_tokens, 96, 512, 2)
    (step,) = seen
    assert checks.step_violations(step, *args) == []
    for slots in ([0, 0], [0, 2], [-1, 0], [0]):
        step.state_slots = torch.tensor(slots, dtype=torch.int32)
        assert any("state slot" in m for m in checks.step_violations(step, *args))


def test_more_requests_than_slots_wait():
    """A given sequence beyond the state slots is refused until another one ends; generation queues."""
    eng = engine("plain", "cpu", torch.float32, max_batch_size=2)
    a, b, c = (eng.open_given() for _ in range(3))
    t, want = truth("plain", 150)
    for sid in (a, b):
        eng.step_given([(sid, t[:9], [])])
    with pytest.raises(RuntimeError, match="state slots"):
        eng.step_given([(c, t[:9], [])])
    eng.close_given(a)
    check(eng.step_given([(c, t[:9], list(range(9)))]).float(), want[:9], torch.float32, "cpu")
    for sid in (b, c):
        eng.close_given(sid)
    prompts = [hlp.tokens(CONFIGS["plain"], n, 80 + n) for n in (9, 5, 14, 3, 8)]
    for p, r in zip(prompts, eng.generate(prompts, greedy(6))):
        assert_greedy("plain", p, r.outputs[0].tokens, torch.float32)
    assert eng.scheduler.check_invariants()[0]


def test_these_tests_would_notice(monkeypatch):
    """The weights make faults visible: each mistake planted in the oracle moves the logits far beyond the 32-bit limit
    (the ops' own tests hold the kernels of both precisions to single keys, experts and states that stand out)."""
    bar = 1000 * LIMIT[torch.float32]
    name = "unequal"
    c, w = CONFIGS[name], weights_of(name)
    t, want = truth(name, 150)

    def planted(edit=None, ww=None):
        cc = copy.deepcopy(c)
        if edit:
            edit(cc)
        return hlp.error(oracle.forward(t, cc, ww or w), want)

    left = lambda cc, i=1: cc["layers"][i]["mixer"]["left"]  # noqa: E731
    assert planted(lambda cc: left(cc)["mask"].update(size=21)) > bar
    assert planted(lambda cc: left(cc)["mask"].update(keep_first=4)) > bar
    assert planted(lambda cc: left(cc, 3)["mask"].update(size=32)) > bar
    assert planted(lambda cc: left(cc).update(bias_max=44)) > bar
    assert planted(lambda cc: left(cc).update(scale=left(c)["scale"] * 1.02)) > bar / 3
    assert planted(lambda cc: cc["layers"][1]["mixer"].update(left_scale=1.26)) > bar / 30
    assert planted(lambda cc: cc["layers"][1]["mixer"].update(right_scale=0.81)) > bar / 30
    assert planted(lambda cc: cc["layers"][0]["mixer"].update(norm_groups=1)) > bar
    assert planted(lambda cc: cc["layers"][0]["mlp"]["router"]["groups"].update(keep=2)) > bar / 3
    assert planted(lambda cc: cc["layers"][0]["mlp"]["router"].update(top=3)) > bar / 3
    assert planted(lambda cc: cc["layers"][0]["mlp"]["expert"].update(limit=1.1)) > bar / 30
    assert planted(lambda cc: cc["embedding"].update(scale=3.1)) > bar / 3
    assert planted(lambda cc: cc.update(logit_softcap=23.0)) > bar / 300
    for key in ("l1.mix.left.pb", "l1.mix.left.q.b", "l0.mix.D", "l0.mix.conv.b", "l2.shift", "l1.shift", "pos"):
        assert planted(None, {**w, key: w[key] * 0}) > bar, key
    for key in ("l0.mix.A_log", "l0.mix.dt_bias", "l1.mix.right.A_log", "l1.mix.right.dt_bias"):
        assert planted(None, {**w, key: w[key].roll(1)}) > bar / 3, key
    plain = oracle.unit
    monkeypatch.setattr(oracle, "unit", lambda x: plain(x) * 1.01)
    assert planted() > bar / 3
    monkeypatch.setattr(oracle, "unit", plain)
    # a state that is lost at token 40
    for fn in ("state_space", "delta_rule"):
        whole = getattr(oracle, fn)
        rows = {"state_space": (0, 1, 2, 3), "delta_rule": (0, 1, 2, 3, 4)}[fn]
        monkeypatch.setattr(oracle, fn, lambda *a: torch.cat([whole(*[x[:40] if i in rows else x for i, x in enumerate(a)]),
                                                              whole(*[x[40:] if i in rows else x for i, x in enumerate(a)])]))
        lost = oracle.forward(t, c, w)
        monkeypatch.setattr(oracle, fn, whole)
        assert hlp.error(lost[41:60], want[41:60]) > bar and hlp.error(lost[-20:], want[-20:]) > bar / 3
