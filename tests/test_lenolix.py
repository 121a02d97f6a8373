"""The Lenolix family through the engine (block pool, scheduler, sampler, trace replay) against the plain equations of
lenolix_oracle: whole prompts, single tokens, portions, mixed batches, reused blocks, generation."""
import copy
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import lenolix_helpers as hlp
import lenolix_oracle as oracle
from decoder_helpers import LIMIT, PLACES, check, greedy, greedy_within_rounding, run_batch
from lenolix_helpers import CONFIGS
from ksanallm_b200.config import EngineConfig, model_config_from_hf
from ksanallm_b200.llm import LLM
from ksanallm_b200.ops import native
from ksanallm_b200.utils import native_engine as ne

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
NAMES = sorted(CONFIGS)


@functools.lru_cache(maxsize=None)
def weights_of(name):
    return hlp.weights(CONFIGS[name], seed=NAMES.index(name))


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
    for sizes in ([150], [1], [2], [40, 1, 2, 17, 3, 1, 1, 30], [15, 2, 47, 3], [100, 1]):
        check(hlp.run_portions(eng, t, sizes), want, dtype, device)
    for n in (1, 2):
        check(hlp.run_portions(eng, t[:n], [n]), want[:n], dtype, device)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_stream_after_every_layer_run(device, dtype):
    name = "unequal"
    t, streams = hlp.tokens(CONFIGS[name], 60, 3), []
    oracle.forward(t, CONFIGS[name], weights_of(name), streams)
    eng = engine(name, device, dtype)
    got = []
    eng.model.stream_hook = lambda r, x: got.append(x.float().cpu().clone())
    hlp.run_portions(eng, t, [60])
    assert len(got) == len(streams) == 5
    for a, b in zip(got, streams):
        assert float((a - b).abs().max() / b.abs().max()) < (1e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_long_decoding(device, dtype):
    """Windows pass over decoded tokens only, across many blocks."""
    n = 330 if device == "cuda" else 200
    t, want = truth("grouped", n, 7)
    eng = engine("grouped", device, dtype)
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
def test_mixed_batches_and_reused_blocks(name, device, dtype):
    lens = (150, 33, 1, 97, 64, 17, 128, 5)
    cases = [truth(name, n, k) for k, n in enumerate(lens)]
    # room for four live requests at a time, far less than for all eight: blocks are handed out again
    eng = engine(name, device, dtype, blocks=31, max_len=160)
    for seed in (0, 1):
        for got, (_, want) in zip(run_batch(eng, [t for t, _ in cases], seed), cases):
            check(got, want, dtype, device)
    st = eng.scheduler.stats()
    assert st["used_blocks"] == 0 and eng.scheduler.check_invariants()[0]


# ------------------------------------------------------------------------------------------------ given-token steps
def test_given_steps_order_and_errors():
    eng = engine("odd", "cpu", torch.float32, blocks=4, max_len=60)
    a, b = eng.open_given(), eng.open_given()
    t, want = truth("odd", 150)
    # a single-token entry first: the plan runs multi-token entries first, the answer keeps the caller's order
    got = eng.step_given([(a, t[:1], [0]), (b, t[:9], [8, 0, 8])])
    check(got, want[[0, 8, 0, 8]], torch.float32, "cpu")
    assert eng.step_given([(a, t[1:2], [])]).shape == (0, 101)
    for bad in ([(a, t[2:4], [2])], [(a, [], [])], [(999, [1], [])], [(a, [1], []), (a, [1], [])], [(b, t[9:70], [])]):
        with pytest.raises(RuntimeError):
            eng.step_given(bad)
    with pytest.raises(RuntimeError, match="blocks"):
        eng.step_given([(a, t[2:40], []), (b, t[9:40], [])])
    check(eng.step_given([(a, t[2:40], [37])]), want[[39]], torch.float32, "cpu")     # the refused steps left nothing behind
    eng.close_given(b)
    check(eng.step_given([(a, t[40:55], [14])]), want[[54]], torch.float32, "cpu")


def test_plans_carry_the_previous_tokens():
    sc = ne.SchedulerConfig()
    sc.max_step_tokens = 20
    s = ne.Scheduler(sc, 16, 0)
    cfg = ne.SamplingConfig()
    cfg.max_new_tokens = 3
    s.add_request(1, list(range(100, 130)), cfg)
    p = s.schedule()
    assert p.prev_ids.tolist() == [-1] + p.input_ids.tolist()[:-1]
    q = ne.StepPlan.unpack(p.pack())
    assert q.prev_ids.tolist() == p.prev_ids.tolist() and q.input_ids.tolist() == p.input_ids.tolist()
    s.advance(p)
    p = s.schedule()                                        # the prompt's second portion
    assert p.input_ids.tolist()[0] == 116 and p.prev_ids.tolist() == list(range(115, 129))
    s.advance(p)
    d = s.schedule()                                        # the sampled token is a placeholder, the one before it is known
    assert d.input_ids.tolist() == [-1] and d.prev_ids.tolist() == [129]


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
    for name in ("unequal", "grouped"):
        eng = engine(name, device, dtype, blocks=80, max_len=200, **options)
        prompts = [hlp.tokens(CONFIGS[name], n, 20 + k) for k, n in enumerate(PROMPTS)]
        for again in range(2):                              # the second time prefixes are cached and blocks reused
            reqs = eng.generate(prompts, greedy(16))
            for p, r in zip(prompts, reqs):
                assert r.status_code == 0 and len(r.outputs[0].tokens) == 16
                if again or len(p) < 40:
                    assert_greedy(name, p, r.outputs[0].tokens, dtype)
        if options.get("enable_auto_prefix_cache"):
            assert eng.scheduler.stats()["prefix_hit_tokens"] > 0
        if options.get("graphs"):
            assert eng.runner.graph_replays > 10
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


@pytest.mark.parametrize("device,dtype", PLACES)
def test_forked_siblings_and_beams(device, dtype):
    """Siblings share the prompt's blocks; the partly filled one is copied, whatever its layers' sizes."""
    name, p = "unequal", hlp.tokens(CONFIGS["unequal"], 37, 50)
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
    best = max(sum(float(torch.log_softmax(row, -1)[t]) for row, t in zip(
        oracle.forward(p + o.tokens[:-1], CONFIGS[name], weights_of(name))[36:], o.tokens)) for o in r.outputs)
    (g,) = eng.generate([p], greedy(12))
    one = sum(float(torch.log_softmax(row, -1)[t]) for row, t in zip(
        oracle.forward(p + g.outputs[0].tokens[:-1], CONFIGS[name], weights_of(name))[36:], g.outputs[0].tokens))
    assert best >= one - 0.5


@pytest.mark.parametrize("device,dtype", PLACES)
def test_moved_keys_are_turned(device, dtype):
    """Copies that land at another position: every layer run's keys turn by the position delta, values stay."""
    name = "unequal"
    eng = engine(name, device, dtype, blocks=20, max_len=160)
    t = hlp.tokens(CONFIGS[name], 32, 1)
    sid = eng.open_given()
    eng.step_given([(sid, t, [])])
    m = eng.model
    src = 1                                                  # any block: whatever it holds turns
    before = m.kv_cache.clone()
    m.kv_cache[9].copy_(m.kv_cache[src])
    m.rerotate_blocks(np.array([[src, 9, 48], [src, src, 0]], dtype=np.int32))
    for run, (k, v) in zip(m.runs, m.panels):
        rot = CONFIGS[name]["layers"][run.layer]["mixer"]["rot"]
        k0, _ = m.layout.views(before, run.cache)
        real = CONFIGS[name]["layers"][run.layer]["mixer"]["dim"]
        want = oracle.rotate(k0[src].float().cpu()[..., :real], 48, oracle.rope_frequencies(rot["dims"], rot["base"], rot["scaling"]))
        assert torch.allclose(k[9].float().cpu()[..., :real], want, atol=1e-5 if dtype == torch.float32 else 0.05)
        assert torch.equal(v[9], m.layout.views(before, run.cache)[1][src]) and torch.equal(k[src], k0[src])


@pytest.mark.parametrize("device,dtype", PLACES)
def test_forward_targets_and_spliced_embeddings(device, dtype):
    """Hidden states, per-position logits and replaced embedding rows of the /forward interface."""
    name = "odd"                                            # width 70: rows are padded inside
    t, want = truth(name, 150)
    eng = engine(name, device, dtype)
    s = greedy(1)
    r = eng.add_request(t[:30], s, request_target={
        "transformer": {"slice_pos": [[3, 5]], "token_reduce_mode": "GATHER_ALL"},
        "logits": {"slice_pos": [[0, 20]], "token_reduce_mode": "GATHER_TOKEN_ID"}})
    while not r.done.is_set():
        eng.step()
    streams = []
    oracle.forward(t[:30], CONFIGS[name], weights_of(name), streams)
    got = r.response["transformer"]
    assert got.shape == (3, 70)
    tol = 1e-4 if dtype == torch.float32 else 0.1
    assert float((got - streams[-1][3:6]).abs().max() / streams[-1].abs().max()) < tol
    probs = torch.softmax(want[:21], -1)[torch.arange(21), torch.tensor(t[1:22])]
    assert torch.allclose(r.response["logits"].reshape(-1), probs, atol=tol)
    # a row spliced over the embedding output: same as a token whose embedding it is
    w = copy.deepcopy(weights_of(name))
    emb = torch.randn(1, 70, generator=torch.Generator().manual_seed(4)).bfloat16().float()
    w["embed_out"] = emb
    a = eng.generate([t[:10]], greedy(1))[0].outputs[0].tokens
    q = eng.add_request(t[:10], greedy(4), refit=([9], [emb * 3]))
    while not q.done.is_set():
        eng.step()
    x = oracle.embed(t[:10], CONFIGS[name], w)
    x[9] = emb[0] * 3
    for i in range(2):
        x = oracle.layer(x, i, CONFIGS[name], w)
    lg = oracle.layer_norm(x, w["final.norm"], w["final.norm.b"], 1e-5) @ w["embed"].t()
    first = q.outputs[0].tokens[0]
    assert float(lg[9].max() - lg[9][first]) <= 0.12 * float(lg.std()) and len(a) == 1


# ------------------------------------------------------------------------------------------------ from a checkpoint
@pytest.mark.parametrize("device,dtype", PLACES)
def test_served_from_a_checkpoint(tmp_path, device, dtype):
    name = "grouped"
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


def test_trace_replay_refuses_what_has_no_32_bit_path(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "llama", "hidden_size": 64, "num_attention_heads": 4}))
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "64"], input="", text=True, capture_output=True, timeout=300)
    assert p.returncode == 3


def test_served_over_http_by_token_ids(tmp_path):
    """The server's entry point from a YAML file, for a checkpoint without a tokenizer."""
    import time
    import urllib.error
    import urllib.request
    import socket
    name = "grouped"
    hlp.save_checkpoint(str(tmp_path / "model"), CONFIGS[name], weights_of(name))
    (tmp_path / "serve.yaml").write_text(
        "setting:\n  batch_scheduler: {max_token_len: 128, max_batch_size: 4}\n"
        "  block_manager: {device_blocks_num: 40, host_blocks_num: 4}\n"
        "model_spec:\n  base_model: {model_dir: model}\n")
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    p = subprocess.Popen([sys.executable, os.path.join(ROOT, "serving_server.py"), "--config_file", str(tmp_path / "serve.yaml"),
                          "--host", "127.0.0.1", "--port", str(port)], env=dict(os.environ, CUDA_VISIBLE_DEVICES=""),
                         stdout=subprocess.DEVNULL, stderr=subprocess.DEVNULL, cwd=str(tmp_path))
    try:
        prompt = hlp.tokens(CONFIGS[name], 20, 80)
        body = json.dumps({"input_tokens": prompt, "sampling_config": {"max_new_tokens": 8, "ignore_eos": True}}).encode()
        for _ in range(120):
            try:
                r = urllib.request.urlopen(urllib.request.Request(f"http://127.0.0.1:{port}/generate", body,
                                                                  {"Content-Type": "application/json"}), timeout=60)
                break
            except (urllib.error.URLError, ConnectionError):
                assert p.poll() is None
                time.sleep(0.5)
        assert_greedy(name, prompt, json.loads(r.read().split(b"\0")[0])["output_token_ids"][0], torch.bfloat16)
    finally:
        p.terminate()
        p.wait(30)


# ------------------------------------------------------------------------------------------------ configuration, loading
def test_configuration_is_read():
    c = model_config_from_hf(copy.deepcopy(CONFIGS["unequal"]))
    assert c.model_type == "lenolix" and c.hidden_size == 72 and c.vocab_size == 203 and c.num_layers == 3
    a = c.layer_specs[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first) == (6, 2, 24, 16, 13, 3)
    assert a.rotary.dims == 8 and a.rotary.scaling["factor"] == 3.0
    assert c.layer_specs[1].mlp is None and c.layer_specs[1].mixer.window == 0
    assert (c.loop.start, c.loop.stop, c.loop.times) == (0, 2, 2) and c.pair_embedding.buckets == 61
    assert model_config_from_hf(copy.deepcopy(CONFIGS["odd"])).loop is None


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][0].update(type="convolution"), lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][0]["mixer"].update(heads=5), lambda c: c["loop"].update(stop=9),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0)])
def test_unknown_configurations_are_refused(edit):
    c = copy.deepcopy(CONFIGS["unequal"])
    edit(c)
    with pytest.raises(ValueError):
        model_config_from_hf(c)


def test_wrong_shapes_and_cache_types_are_refused():
    w = dict(weights_of("unequal"))
    w["l0.mix.k"] = w["l0.mix.k"][:-1]
    with pytest.raises(ValueError, match="l0.mix.k"):
        hlp.build(CONFIGS["unequal"], w, "cpu", torch.float32)
    m = hlp.build(CONFIGS["unequal"], weights_of("unequal"), "cpu", torch.float32)
    with pytest.raises(ValueError):
        m.allocate_kv_cache(4, 16, torch.float8_e4m3fn)


def test_these_tests_would_notice():
    """The weights make faults visible: each mistake planted in the oracle moves the logits far beyond the 32-bit limit
    (the ops' own tests hold the kernels of both precisions to single keys that stand out)."""
    bar = 1000 * LIMIT[torch.float32]
    for name in ("unequal", "grouped"):
        c, w = CONFIGS[name], weights_of(name)
        t, want = truth(name, 150)

        def planted(edit, ww=None):
            cc = copy.deepcopy(c)
            if edit:
                edit(cc)
            return hlp.error(oracle.forward(t, cc, ww or w), want)

        mask = [i for i, e in enumerate(c["layers"]) if e["mixer"]["mask"]]
        for i in mask:
            assert planted(lambda cc: cc["layers"][i]["mixer"]["mask"].update(size=c["layers"][i]["mixer"]["mask"]["size"] + 1)) > bar
            assert planted(lambda cc: cc["layers"][i]["mixer"]["mask"].update(keep_first=c["layers"][i]["mixer"]["mask"]["keep_first"] - 1)) > bar
        assert planted(lambda cc: cc["embedding"]["bigram"].update(mul_prev=0)) > bar
        assert planted(lambda cc: cc["layers"][0]["mixer"]["rot"].update(scaling=None)) > bar
        assert planted(None, {k: v for k, v in w.items() if not k.endswith("sink")}) > bar
        assert planted(None, {**w, "loop.step": w["loop.step"].flip(0)}) > bar


# ------------------------------------------------------------------------------------------------ several ranks
@pytest.mark.parametrize("name,world", [("grouped", 2), ("wide2", 2), ("unequal4", 4)])
def test_tensor_parallel_shards(tmp_path, name, world):
    """Heads, feed-forward columns and the vocabulary split over ranks (key/value heads shared where there are fewer)."""
    import socket
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    out = str(tmp_path / "logits.pt")
    r = subprocess.run([sys.executable, "-m", "torch.distributed.run", "--nnodes=1", f"--nproc-per-node={world}", "--master-addr",
                        "127.0.0.1", "--master-port", str(port), os.path.join(ROOT, "tests", "stream_tp_worker.py"), out, "lenolix", name],
                       env=dict(os.environ, CUDA_VISIBLE_DEVICES="", OMP_NUM_THREADS="2"), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-3000:]
    c = hlp.SPLIT.get(name) or CONFIGS[name]
    check(torch.load(out), oracle.forward(hlp.tokens(c, 60), c, hlp.weights(c, 3)), torch.float32, "cpu")


def test_layouts_that_cannot_be_split_are_refused():
    from ksanallm_b200.models.weights import DictSource, build_model
    cfg = model_config_from_hf(copy.deepcopy(CONFIGS["odd"]))
    with pytest.raises(ValueError):
        build_model(cfg, DictSource(weights_of("odd"), "lenolix"), 0, 2)
    with pytest.raises(ValueError):
        build_model(cfg, DictSource(weights_of("odd"), "lenolix"), layer_range=(0, 0))
