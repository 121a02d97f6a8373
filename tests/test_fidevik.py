"""The Fidevik family through the engine (block pool, scheduler, sampler, trace replay) against the plain equations of
fidevik_oracle: whole prompts, single tokens, portions, mixed batches, reused blocks, generation."""
import copy
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import fidevik_helpers as hlp
import fidevik_oracle as oracle
from decoder_helpers import LIMIT, PLACES, check, greedy, greedy_within_rounding, run_batch
from fidevik_helpers import CONFIGS
from ksanallm_b200.config import AttentionSpec, EngineConfig, GatedMlpSpec, LatentAttentionSpec, MoeSpec, model_config_from_hf
from ksanallm_b200.llm import LLM
from ksanallm_b200.models.weights import DictSource, build_model
from ksanallm_b200.ops import native

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
    for sizes in ([150], [2], [40, 1, 2, 17, 3, 1, 1, 30], [15, 2, 47, 3], [100, 1], [16]):
        check(hlp.run_portions(eng, t, sizes), want, dtype, device)
    short = 150 if device == "cuda" else 50
    check(hlp.run_portions(eng, t[:short], [1]), want[:short], dtype, device)
    for n in (1, 2, 16, 17):
        check(hlp.run_portions(eng, t[:n], [n]), want[:n], dtype, device)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("name", ["unequal", "odd", "ones"])
def test_stream_after_every_layer_run(name, device, dtype):
    t, streams = hlp.tokens(CONFIGS[name], 60, 3), []
    oracle.forward(t, CONFIGS[name], weights_of(name), streams)
    eng = engine(name, device, dtype)
    got = []
    eng.model.stream_hook = lambda r, x: got.append(x[:, :CONFIGS[name]["width"]].float().cpu().clone())
    hlp.run_portions(eng, t, [60])
    assert len(got) == len(streams) == len(oracle.order(CONFIGS[name]))
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
def test_mixed_batches_and_reused_blocks(name, device, dtype):
    lens = (150, 33, 1, 97, 64, 17, 128, 5)
    cases = [truth(name, n, k) for k, n in enumerate(lens)]
    # room for four live requests at a time, far less than for all eight: blocks are handed out again
    eng = engine(name, device, dtype, blocks=31, max_len=160)
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
def test_moved_blocks_of_the_flexible_cache(device, dtype):
    """A cached stretch behind another first block: approximate by design, so only the service is checked here (the turned keys
    are held to the equations in the ops' tests)."""
    name = "unequal"
    eng = engine(name, device, dtype, blocks=80, max_len=200, enable_auto_prefix_cache=True, min_flexible_cache_num=16)
    base = hlp.tokens(CONFIGS[name], 64, 70)
    eng.generate([base], greedy(4))
    (r,) = eng.generate([hlp.tokens(CONFIGS[name], 16, 71) + base[16:]], greedy(8))
    assert r.status_code == 0 and len(r.outputs[0].tokens) == 8
    assert eng.scheduler.check_invariants()[0]
    if device == "cuda":
        native.check_err_flag("cuda")


@pytest.mark.parametrize("device,dtype", PLACES)
def test_forward_targets_and_spliced_embeddings(device, dtype):
    """Hidden states, per-position logits and replaced embedding rows of the /forward interface. The spliced row is also what
    later passes of the loop add again."""
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
    w = dict(weights_of(name))
    w["embed"] = torch.cat([w["embed"], emb])
    rows = oracle.forward(t[:9] + [101], c, w)[:, :101]
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
    assert (c.model_type, c.hidden_size, c.vocab_size, c.num_layers) == ("fidevik", 72, 203, 5)
    assert (c.logit_scale, c.rms_norm_eps, c.tie_word_embeddings) == (0.7, 1e-5, False)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 4, 3)
    a, b = c.layer_specs[0].mixer, c.layer_specs[1].mixer
    assert isinstance(a, LatentAttentionSpec) and (a.heads, a.dim, a.vdim, a.q_rank, a.kv_rank) == (3, 16, 24, 24, 40)
    assert a.sink and a.head_gate and a.rotary is None and a.window == 0
    assert isinstance(b, AttentionSpec) and (b.heads, b.kv_heads, b.dim, b.vdim) == (6, 2, 24, 16)
    assert (b.rotary.dims, b.rotary.base, b.rotary.interleaved) == (8, 500.0, True) and b.qk_norm and not b.sink
    f, e = c.layer_specs[0].mlp, c.layer_specs[1].mlp
    assert isinstance(f, GatedMlpSpec) and (f.size, f.act) == (40, "gelu") and c.layer_specs[2].mlp is None
    assert isinstance(e, MoeSpec) and (e.router.experts, e.router.top, e.router.groups, e.router.keep_groups) == (12, 4, 4, 2)
    assert (e.expert.size, e.expert.act, e.shared.size) == (24, "silu", 40) and not e.router.renorm
    p = model_config_from_hf(copy.deepcopy(CONFIGS["plain"]))
    assert p.loop is None and p.layer_specs[0].mixer.rotary is None


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][0].update(type="convolution"), lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][1]["mixer"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), lambda c: c["layers"][0]["mixer"].update(q_rank=0),
    lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5), lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7), lambda c: c["loop"].update(stop=6), lambda c: c["loop"].update(start=4),
    lambda c: c["loop"].update(times=0), lambda c: c.update(layers=[])])
def test_unknown_configurations_are_refused(edit):
    c = copy.deepcopy(CONFIGS["unequal"])
    edit(c)
    with pytest.raises(ValueError):
        model_config_from_hf(c)


def test_wrong_shapes_and_unsupported_options_are_refused():
    name = "unequal"
    for key in ("l0.mix.uq", "l1.mlp.e3.down", "l1.mix.q.norm", "loop.step"):
        w = dict(weights_of(name))
        w[key] = w[key][:-1]
        with pytest.raises(ValueError, match=key):
            hlp.build(CONFIGS[name], w, "cpu", torch.float32)
    m = hlp.build(CONFIGS[name], weights_of(name), "cpu", torch.float32)
    assert m.weight_bytes() > 0
    with pytest.raises(ValueError):
        m.allocate_kv_cache(4, 16, torch.float8_e4m3fn)
    cfg = model_config_from_hf(copy.deepcopy(CONFIGS["odd"]))
    with pytest.raises(ValueError):
        build_model(cfg, DictSource(weights_of("odd"), "fidevik"), 0, 2)
    with pytest.raises(ValueError):
        build_model(cfg, DictSource(weights_of("odd"), "fidevik"), layer_range=(0, 0))


def test_these_tests_would_notice(monkeypatch):
    """The weights make faults visible: each mistake planted in the oracle moves the logits far beyond the 32-bit limit
    (the ops' own tests hold the kernels of both precisions to single keys, experts and sinks that stand out)."""
    bar = 1000 * LIMIT[torch.float32]
    name = "unequal"
    c, w = CONFIGS[name], weights_of(name)
    t, want = truth(name, 150)

    def planted(edit=None, ww=None):
        cc = copy.deepcopy(c)
        if edit:
            edit(cc)
        return hlp.error(oracle.forward(t, cc, ww or w), want)

    assert planted(lambda cc: cc["layers"][1]["mixer"]["rot"].update(base=505.0)) > bar / 30
    assert planted(lambda cc: cc["layers"][1]["mixer"]["rot"].update(dims=6)) > bar
    assert planted(lambda cc: cc["layers"][1]["mlp"]["router"]["groups"].update(keep=3)) > bar / 3
    assert planted(lambda cc: cc["layers"][1]["mlp"]["router"].update(top=3)) > bar / 3
    assert planted(lambda cc: cc["loop"].update(times=2)) > bar
    assert planted(lambda cc: cc.update(logit_scale=0.71)) > bar / 3
    for i in (0, 2, 4):
        assert planted(lambda cc: cc["layers"][i]["mixer"].update(scale=c["layers"][i]["mixer"]["scale"] * 1.02)) > bar / 30
        assert planted(None, {**w, f"l{i}.mix.sink": w[f"l{i}.mix.sink"] - 100}) > bar
    assert planted(None, {**w, "l1.mlp.correction": w["l1.mlp.correction"] * 0}) > bar / 3
    assert planted(None, {**w, "loop.step": w["loop.step"].flip(0)}) > bar
    assert planted(None, {**w, "l1.mix.q.norm": w["l1.mix.q.norm"].roll(24)}) > bar
    plain = oracle.rms_norm
    for part in (8, 24):                                     # norms per head instead of over the whole projection
        monkeypatch.setattr(oracle, "rms_norm", lambda x, g, eps: plain(x.unflatten(-1, (-1, part)), 1.0, eps).flatten(-2) * g
                            if x.shape[-1] in (144, 48) else plain(x, g, eps))
        assert planted() > bar
    monkeypatch.setattr(oracle, "rms_norm", plain)
    early = oracle.forward(t[1:], c, w)                      # the first key is missing
    assert hlp.error(early[-50:], want[-50:]) > bar / 3


# ------------------------------------------------------------------------------------------------ several ranks
@pytest.mark.parametrize("name,world", [("split2", 2), ("split4", 4)])
def test_tensor_parallel_shards(tmp_path, name, world):
    """Heads (key heads on several ranks among them), feed-forward and expert columns and the vocabulary split over ranks, norms
    over the whole projections, latents replicated."""
    import socket
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        port = s.getsockname()[1]
    out = str(tmp_path / "logits.pt")
    r = subprocess.run([sys.executable, "-m", "torch.distributed.run", "--nnodes=1", f"--nproc-per-node={world}", "--master-addr",
                        "127.0.0.1", "--master-port", str(port), os.path.join(ROOT, "tests", "stream_tp_worker.py"), out, "fidevik", name],
                       env=dict(os.environ, CUDA_VISIBLE_DEVICES="", OMP_NUM_THREADS="2"), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-3000:]
    c = hlp.SPLIT[name]
    check(torch.load(out), oracle.forward(hlp.tokens(c, 60), c, hlp.weights(c, 3)), torch.float32, "cpu")
