"""The mechanisms of the Lenolix family one by one: the ops (plain statements on the CPU, kernels on the GPU) against
the plain equations of lenolix_oracle."""
import math
from types import SimpleNamespace

import pytest
import torch

import lenolix_oracle as oracle
from lenolix_helpers import PLACES, ROTATION
from ksanallm_b200.models.common import PanelLayout
from ksanallm_b200.ops import dispatch as ops
from ksanallm_b200.ops import native
from ksanallm_b200.ops import reference as ref

TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}
rand = lambda seed, *s: torch.randn(*s, generator=torch.Generator().manual_seed(seed)).bfloat16().float()  # noqa: E731


def close(got, want, dtype, scale=None):
    got, want = got.float().cpu(), want.float()
    s = scale if scale is not None else max(1.0, float(want.abs().max()))
    assert torch.isfinite(got).all()
    assert float((got - want).abs().max()) <= TOL[dtype] * s, float((got - want).abs().max()) / s


# ------------------------------------------------------------------------------------------------ embedding
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("hashed", [None, (61, 7, 3), (1, 1, 1), (499, 2147483647, 999999937)])
def test_pair_embedding(device, dtype, hashed):
    V, W = 203, 72
    cfg = {"embedding": {"scale": 3.5}}
    w = {"embed": rand(0, V, W)}
    if hashed:
        cfg["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), hashed))
        w["bigram"] = rand(1, hashed[0] + 1, W)
    toks = torch.randint(0, V, (50,), generator=torch.Generator().manual_seed(2)).tolist()
    want = oracle.embed(toks, cfg, w)
    ids = torch.tensor(toks, dtype=torch.int32, device=device)
    prev = torch.tensor([-1] + toks[:-1], dtype=torch.int32, device=device)
    copy = torch.zeros(50, 2 * W, dtype=dtype, device=device)
    x = ops.embed_pair(ids, prev, w["embed"].to(device, dtype), w["bigram"].to(device, dtype) if hashed else None, 3.5,
                       *(hashed or (0, 0, 0)), copy=copy[:, W:])
    assert x.dtype == torch.float32
    close(x, want, torch.float32)                  # the stream is 32-bit whatever the activations' type
    close(copy[:, W:], want, dtype)
    assert not copy[:, :W].any()


# ------------------------------------------------------------------------------------------------ norms
def norm_params(H, HP, seed, device, dtype, eps, rms=False):
    w, b = rand(seed, H), rand(seed + 1, H)
    pad = lambda t: torch.nn.functional.pad(t, (0, HP - H)).to(device, dtype)  # noqa: E731
    return ops.NormParams(pad(w), None if rms else pad(b), H, eps, rms), w, b


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H", [64, 70, 201, 2056, 8200])
def test_sandwich_norm(device, dtype, H):
    HP, M, eps = (H + 7) // 8 * 8, 7, 0.3
    x, y = rand(0, M, H) * 30 + 1000, rand(1, M, H) * 0.05 + 0.5      # a large mean, a small spread: cancellation shows
    post, w1, b1 = norm_params(H, HP, 2, device, dtype, eps)
    then, w2, b2 = norm_params(H, HP, 4, device, dtype, eps)
    ls = rand(6, H)
    pad = lambda t, d: torch.nn.functional.pad(t, (0, HP - H)).to(device, d)  # noqa: E731
    y = y.to(dtype).float()
    want_x = x.double() + oracle.layer_norm(y.double(), w1.double(), b1.double(), eps) * ls.double()
    want_z = oracle.layer_norm(want_x, w2.double(), b2.double(), eps)
    xs = pad(x, torch.float32)
    out, z = ops.stream_add(xs, pad(y, dtype), post, pad(ls, dtype), then)
    assert out.data_ptr() == xs.data_ptr() and z.dtype == dtype
    # fp32 rounding of the stream itself (values near 1000) is 6e-5
    assert float((out[:, :H].double().cpu() - want_x).abs().max()) < 3e-4
    close(z[:, :H], want_z, dtype, scale=10)
    assert not out[:, H:].any() and not z[:, H:].any()
    # the norm alone, a gather, a copy into a strided buffer, and an add that leaves its input alone
    rows = torch.tensor([5, 0, 5], dtype=torch.int32, device=device)
    close(ops.stream_norm(xs, then, dtype, rows=rows)[:, :H], want_z[[5, 0, 5]], dtype, scale=10)
    buf = torch.zeros(M, 2 * HP, dtype=dtype, device=device)
    before = xs.clone()
    out2, z2 = ops.stream_add(xs, pad(y, dtype), post, pad(ls, dtype), None, buf[:, :HP], inplace=False)
    assert z2 is None and torch.equal(xs, before) and out2.data_ptr() != xs.data_ptr()
    close(buf[:, :HP], out2.cpu(), dtype, scale=2000)
    assert not buf[:, HP:].any()


@pytest.mark.parametrize("device,dtype", PLACES)
def test_rms_variant_and_plain_add(device, dtype):
    H, M = 136, 5
    x, y = rand(0, M, H), rand(1, M, H)
    n, w, _ = norm_params(H, H, 2, device, dtype, 1e-6, rms=True)
    rms = lambda t: t / torch.sqrt((t * t).mean(-1, keepdim=True) + 1e-6) * w  # noqa: E731
    close(ops.stream_norm(x.to(device), n, dtype), rms(x), dtype)
    out, z = ops.stream_add(x.clone().to(device), y.to(device, dtype), None, None, n)
    close(out, x + y, torch.float32)
    close(z, rms(x + y), dtype)


# ------------------------------------------------------------------------------------------------ gated unit
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("limit", [0.5, 7.0])
def test_clamped_unit(device, dtype, limit):
    W, ff = 16, 24
    w = {"gate": rand(0, ff, W), "up": rand(1, ff, W), "down": torch.eye(ff)}
    h = rand(2, 200, W)
    gu = torch.cat([h @ w["gate"].t(), h @ w["up"].t()], 1).to(dtype)
    # the identity as down projection: the oracle's result is the unit's; its input is what the unit reads
    ident = {"gate": torch.eye(ff, 2 * ff), "up": torch.cat([torch.zeros(ff, ff), torch.eye(ff)], 1), "down": torch.eye(ff)}
    want = oracle.feed_forward(gu.float(), {"limit": limit}, ident, "")
    close(ops.glu_clamp(gu.to(device), limit), want, dtype)


# ------------------------------------------------------------------------------------------------ rotation + append
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("Hq,Hkv,D,Dv,rot,scaling", [(4, 2, 32, 32, 32, None), (6, 3, 48, 16, 32, ROTATION["scaling"]),
                                                     (3, 1, 24, 40, 14, None), (2, 2, 64, 64, 2, ROTATION["scaling"]),
                                                     (1, 1, 16, 8, 0, None), (8, 2, 128, 128, 80, ROTATION["scaling"])])
def test_partial_rotation_and_append(device, dtype, Hq, Hkv, D, Dv, rot, scaling):
    bt, blocks, base = 16, 5, 300.0
    hf = None if scaling is None else {"rope_type": "llama3", "factor": scaling["factor"], "low_freq_factor": scaling["low"],
                                       "high_freq_factor": scaling["high"], "original_max_position_embeddings": scaling["original"]}
    table = ref.build_cos_sin_cache(rot, 400, base, hf, device) if rot else None
    positions = [0, 1, 17, 63, 64, 399, 5]
    slots = [3, 16, 79, 0, 40, 41, -1]                            # the last row is padding: not written
    qkv = rand(0, 7, (Hq + Hkv) * D + Hkv * Dv)
    layout = PanelLayout([(1, 8, 8), (Hkv, D, Dv)], bt)
    cache = torch.full((blocks, layout.record), 7.0, dtype=dtype, device=device)
    k, v = layout.views(cache, 1)
    dev = qkv.clone().to(device, dtype)
    i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)  # noqa: E731
    ops.qkv_rope_append(dev, i32(positions), i32(slots), table, k, v, bt, Hq, Hkv, rot)
    fr = oracle.rope_frequencies(rot, base, scaling)
    want_k = torch.full(k.shape, 7.0)
    want_v = torch.full(v.shape, 7.0)
    for r, (p, s) in enumerate(zip(positions, slots)):
        q = oracle.rotate(qkv[r, :Hq * D].view(Hq, D), p, fr)
        close(dev[r, :Hq * D].view(Hq, D), q, dtype)
        if s >= 0:
            want_k[s // bt, :, s % bt] = oracle.rotate(qkv[r, Hq * D:(Hq + Hkv) * D].view(Hkv, D), p, fr)
            want_v[s // bt, :, s % bt] = qkv[r, (Hq + Hkv) * D:].view(Hkv, Dv)
    close(k, want_k, dtype)
    close(v, want_v, dtype)
    a, b = layout.views(cache, 0)
    assert bool((a == 7).all()) and bool((b == 7).all())


def test_frequency_scaling_covers_all_three_ranges():
    sc, dims, base = ROTATION["scaling"], 16, ROTATION["base"]
    plain, scaled = oracle.rope_frequencies(dims, base, None), oracle.rope_frequencies(dims, base, sc)
    ratio = [b / a for a, b in zip(plain, scaled)]
    assert any(r == 1 for r in ratio) and any(abs(r - 1 / sc["factor"]) < 1e-12 for r in ratio)
    assert any(1 / sc["factor"] + 1e-6 < r < 1 - 1e-6 for r in ratio)


# ------------------------------------------------------------------------------------------------ attention
def attention_case(H, G, D, Dv, window, keep, lens, bt, device, dtype, seed=0, sink_size=2.0):
    """Sequences of (cached, new) tokens in shuffled blocks. Every query points at one key (its own, the last inside and
    the first outside the window, the last kept and the first not kept token, page and tile borders, a random one), with
    a score that stands out by about 12, so that a key wrongly seen or missed turns the output over."""
    g = torch.Generator().manual_seed(seed)
    scale = D ** -0.5 * 1.3
    order = sorted(range(len(lens)), key=lambda s: lens[s][1] == 1)      # multi-token sequences first
    lens = [lens[s] for s in order]
    nblk = [(p + n + bt - 1) // bt for p, n in lens]
    ids = torch.randperm(sum(nblk) + 3, generator=g).tolist()
    layout = PanelLayout([(G, D, Dv), (1, 8, 16)], bt)
    cache = torch.randn(len(ids), layout.record, generator=g).mul_(3).to(dtype).to(device)    # stale values everywhere
    kc, vc = layout.views(cache, 0)
    table = torch.zeros(len(lens), max(nblk) + 1, dtype=torch.int32)
    sinks = torch.randn(H, generator=g) * sink_size
    qs, want, at = [], [], 0
    for s, (past, n) in enumerate(lens):
        T = past + n
        k = torch.randn(T, G, D, generator=g).to(dtype).float()
        v = torch.randn(T, G, Dv, generator=g).to(dtype).float()
        q = torch.randn(T, H, D, generator=g) * 0.5
        for i in range(T):
            for h in range(H):
                edges = [i, i - window + 1, i - window, keep - 1, keep, i // 16 * 16 - 1, i // 64 * 64, 0,
                         int(torch.randint(0, i + 1, (1,), generator=g))]
                j = edges[(i + 5 * h) % len(edges)]
                if 0 <= j <= i:
                    kj = k[j, h // (H // G)]
                    q[i, h] = kj * (12.0 / (scale * float(kj @ kj)))
        q = q.to(dtype).float()
        mask = {"size": window, "keep_first": keep} if window else None
        o = torch.stack([oracle.attend(q[:, h], k[:, h // (H // G)], v[:, h // (H // G)], sinks[h], scale, mask)
                         for h in range(H)], 1)
        blk = ids[at:at + nblk[s]]
        at += nblk[s]
        table[s, :nblk[s]] = torch.tensor(blk, dtype=torch.int32)
        for t in range(T):
            kc[blk[t // bt], :, t % bt] = k[t].to(device, dtype)
            vc[blk[t // bt], :, t % bt] = v[t].to(device, dtype)
        qs.append(q[past:])
        want.append(o[past:])
    q = torch.cat(qs).reshape(-1, H * D)
    qkv = torch.cat([q, torch.full((q.shape[0], G * (D + Dv)), 9.0)], 1).to(device, dtype)
    news = [n for _, n in lens]
    cu = torch.tensor([0] + news).cumsum(0).to(torch.int32)
    multi = sum(n > 1 for n in news)
    kv = torch.tensor([p + n for p, n in lens], dtype=torch.int32)
    step = SimpleNamespace(block_table=table.to(device), cu_q=cu.to(device), kv_lens=kv.to(device), num_multi=multi,
                           num_single=len(news) - multi, num_multi_tokens=int(cu[multi]), max_q_len=max(news), max_kv_len=int(kv.max()))
    got = ops.panel_attention(qkv, kc, vc, bt, step, H, G, scale, window, keep, sinks.to(device))
    return got.view(-1, H, Dv), torch.cat(want)


LENS = [(0, 1), (0, 150), (63, 2), (64, 1), (130, 70), (127, 1), (200, 3), (15, 17), (255, 1), (31, 33)]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,G,D,Dv,window,keep,bt", [
    (4, 2, 32, 32, 40, 5, 16), (6, 2, 40, 24, 64, 16, 16), (8, 1, 128, 128, 65, 63, 16), (4, 1, 96, 96, 63, 20, 16),
    (3, 3, 64, 96, 100, 0, 16), (3, 1, 24, 16, 17, 1, 8), (24, 1, 64, 64, 30, 70, 32), (2, 1, 136, 72, 33, 4, 16),
    (2, 2, 256, 200, 128, 129, 16), (5, 1, 16, 8, 1, 0, 16), (4, 4, 64, 64, 0, 0, 16), (8, 2, 80, 128, 129, 3, 64),
    (4, 2, 48, 48, 1000, 2, 16), (2, 1, 192, 192, 50, 10, 4)])
def test_window_attention(device, dtype, H, G, D, Dv, window, keep, bt):
    lens = LENS if device == "cuda" else LENS[:1] + LENS[3:8]
    got, want = attention_case(H, G, D, Dv, window, keep, lens, bt, device, dtype)
    close(got, want, dtype, scale=4 if dtype == torch.bfloat16 else None)
    if device == "cuda":
        native.check_err_flag("cuda")


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("window", [0, 300])
def test_window_attention_far_keys(device, dtype, window):
    """Hundreds of keys, a single one of which matters; long enough for several split ranges of the decode kernel."""
    lens = [(900, 1), (640, 1), (1, 2)] + ([(700, 130), (1023, 1), (1, 1)] if device == "cuda" else [])
    got, want = attention_case(4, 2, 64, 64, window, 7, lens, 16, device, dtype, seed=3)
    close(got, want, dtype, scale=4 if dtype == torch.bfloat16 else None)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("size", [0.0, 40.0])
def test_sink_sizes(device, dtype, size):
    """Sinks far above every score empty the row, sinks far below leave a plain softmax."""
    got, want = attention_case(4, 2, 32, 32, 20, 3, [(0, 40), (50, 1), (7, 9)], 16, device, dtype, seed=5, sink_size=size)
    close(got, want, dtype, scale=4 if dtype == torch.bfloat16 else None)
    if size:
        assert float(want.abs().amax(-1).min()) < 1e-3 < float(want.abs().amax(-1).max())


@pytest.mark.gpu
@pytest.mark.parametrize("D,Dv,G", [(96, 96, 4), (128, 64, 2), (64, 128, 8)])
def test_both_prefill_kernels_agree(D, Dv, G, monkeypatch):
    for tc in (True, False):
        monkeypatch.setattr(native, "PREFILL_TC", tc)
        got, want = attention_case(G, 1, D, Dv, 90, 33, [(0, 260), (100, 150), (5, 2)], 16, "cuda", torch.bfloat16, seed=9)
        close(got, want, torch.bfloat16, scale=4)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_no_sink_no_window_equals_plain_softmax(device, dtype):
    g = torch.Generator().manual_seed(0)
    H, D, T, bt = 2, 16, 20, 16
    q, k, v = (torch.randn(T, H, D, generator=g).to(dtype).float() for _ in range(3))
    layout = PanelLayout([(H, D, D)], bt)
    cache = torch.zeros(2, layout.record, dtype=dtype, device=device)
    kc, vc = layout.views(cache, 0)
    for t in range(T):
        kc[t // bt, :, t % bt], vc[t // bt, :, t % bt] = k[t].to(device, dtype), v[t].to(device, dtype)
    qkv = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1).to(device, dtype)
    i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)  # noqa: E731
    step = SimpleNamespace(block_table=i32([[0, 1]]), cu_q=i32([0, T]), kv_lens=i32([T]), num_multi=1, num_single=0,
                           num_multi_tokens=T, max_q_len=T, max_kv_len=T)
    got = ops.panel_attention(qkv, kc, vc, bt, step, H, H, 0.25)
    want = torch.stack([oracle.attend(q[:, h], k[:, h], v[:, h], None, 0.25, None) for h in range(H)], 1).reshape(T, -1)
    close(got, want, dtype)


# ------------------------------------------------------------------------------------------------ fp32 GEMM
@pytest.mark.gpu
@pytest.mark.parametrize("M,N,K", [(1, 8, 8), (63, 130, 72), (200, 64, 1000)])
def test_gemm_f32(M, N, K):
    x, w, b, r = rand(0, M, K), rand(1, N, K), rand(2, N), rand(3, M, N)
    got = native.gemm_f32(x.cuda(), w.cuda(), bias=b.cuda(), residual=r.cuda())
    want = x.double() @ w.double().t() + b.double() + r.double()
    assert float((got.double().cpu() - want).abs().max()) < 1e-5 * math.sqrt(K)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_stream_rows_replaced(device, dtype):
    x = rand(0, 6, 72).to(device)
    keep, emb = x.clone(), rand(1, 2, 70).to(device)
    ops.refit_stream_rows(x, torch.tensor([4, 1], dtype=torch.int32, device=device), emb)
    assert torch.equal(x[[4, 1], :70], emb) and torch.equal(x[[0, 2, 3, 5]], keep[[0, 2, 3, 5]])
    assert torch.equal(x[:, 70:], keep[:, 70:])


@pytest.mark.gpu
def test_bad_indices_are_reported_not_followed():
    """Host-side bookkeeping errors reach the kernels as indices outside their tables: recorded and skipped."""
    table = rand(0, 16, 32).cuda().bfloat16()
    native.clear_err_flag("cuda")
    ops.embed_pair(torch.tensor([3, 16], dtype=torch.int32, device="cuda"), None, table, None, 1.0)
    with pytest.raises(RuntimeError):
        native.check_err_flag("cuda")
    layout = PanelLayout([(1, 16, 16)], 16)
    cache = torch.zeros(2, layout.record, dtype=torch.bfloat16, device="cuda")
    k, v = layout.views(cache, 0)
    i32 = lambda t: torch.tensor(t, dtype=torch.int32, device="cuda")  # noqa: E731
    ops.qkv_rope_append(torch.ones(1, 48, dtype=torch.bfloat16, device="cuda"), i32([0]), i32([32]), None, k, v, 16, 1, 1, 0)
    with pytest.raises(RuntimeError):
        native.check_err_flag("cuda")
    assert not cache.any()
