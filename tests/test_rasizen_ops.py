"""The mechanisms of the Rasizen family one by one: the ops (plain statements on the CPU, kernels on the GPU) against the
plain equations of rasizen_oracle."""
import math
from types import SimpleNamespace

import pytest
import torch

import rasizen_oracle as oracle
from decoder_helpers import PLACES, close, make_step, pad, rand, TOL, up8
from ksanallm_b200.models.common import RecordLayout
from ksanallm_b200.ops import dispatch as ops
from ksanallm_b200.ops import native
from ksanallm_b200.ops import reference as ref


# ------------------------------------------------------------------------------------------------ norms and units
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,groups", [(64, 1), (64, 2), (72, 3), (70, 5), (70, 70), (66, 2), (2048, 4), (2304, 9), (8192, 2), (9000, 1000)])
def test_grouped_norm_with_scaled_residual(device, dtype, H, groups):
    HP, M, eps, alpha = up8(H), 5, 0.02, 0.37
    # parts of very different size: one common root mean square would drown the small ones
    x = rand(0, M, H) * torch.logspace(-2, 2, groups).repeat_interleave(H // groups)
    y, w = rand(1, M, H), rand(2, H)
    n = ops.NormParams(pad(w, HP).to(device, dtype), None, H, eps, rms=True, groups=groups)
    want_x = x.double() + alpha * y.double()
    want_z = oracle.group_norm(want_x, w.double(), groups, eps)
    xs = pad(x, HP).to(device)
    out, z = ops.stream_add(xs, pad(y, HP).to(device, dtype), None, None, n, alpha=alpha)
    assert out.data_ptr() == xs.data_ptr() and z.dtype == dtype
    assert float((out[:, :H].double().cpu() - want_x).abs().max()) < 3e-5 * 4
    close(z[:, :H], want_z, dtype, scale=4)
    assert not out[:, H:].any() and not z[:, H:].any()
    rows = torch.tensor([4, 0, 4], dtype=torch.int32, device=device)
    close(ops.stream_norm(xs, n, dtype, rows=rows)[:, :H], want_z[[4, 0, 4]], dtype, scale=4)
    out, z = ops.stream_add(pad(x, HP).to(device), pad(y, HP).to(device, dtype), None, None, None, alpha=alpha)
    assert z is None and float((out[:, :H].double().cpu() - want_x).abs().max()) < 3e-5 * 4


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("p,q", [(0.8, 0.8), (-1.5, 2.0), (0.0, -30.0), (25.0, -3.0)])
def test_piecewise_unit(device, dtype, p, q):
    x = torch.cat([rand(0, 50, 24) * 4, torch.tensor([[0.0, -0.0, 1e-4, -1e-4, -1e-2, -0.5, -30.0, -90.0] * 3])]).to(dtype)
    want = oracle.xielu(x.double(), p, q)
    got = ops.xielu(x.to(device), oracle.softplus(p), 0.5 + oracle.softplus(q))
    # the two parts of the lower branch may cancel: errors are relative to the larger of them
    assert float(((got.double().cpu() - want).abs() / (want.abs() + x.double().abs() + 1e-3)).max()) < TOL[dtype]


# ------------------------------------------------------------------------------------------------ recurrence
def recurrence_inputs(T, W, seed, dtype):
    """Gates from wide open to nearly shut (the state of a shut channel carries the first tokens for hundreds of steps),
    candidates on both sides of zero and exactly zero."""
    z = rand(seed, T, W) * 1.5 + torch.linspace(-9, 3, W)
    u = rand(seed + 1, T, W) * 2
    u[::7] = 0.0
    u[:3] = 40.0                                        # the first tokens leave a mark that only memory explains
    return [t.to(dtype).float() for t in (z, u, rand(seed + 2, T, W))]


def run_recurrence(W, lens, bt, device, dtype, portions=None, seed=0):
    """Sequences of the given lengths in shuffled blocks of a record layout, each fed in its own portions; outputs per
    sequence and what the oracle says."""
    g = torch.Generator().manual_seed(seed)
    layout = RecordLayout(dtype)
    layout.add((3, 5))
    at = layout.add((W,), torch.float32)
    nblk = [(n + bt - 1) // bt for n in lens]
    ids = torch.randperm(sum(nblk) + 2, generator=g).tolist()
    cache = torch.full((len(ids), layout.record), 7.0, dtype=dtype, device=device)       # stale values everywhere
    state = layout.view(cache, at)
    assert state.dtype == torch.float32 and tuple(state.shape) == (len(ids), W)
    tables, k = [], 0
    for n in nblk:
        tables.append(ids[k:k + n])
        k += n
    data = [recurrence_inputs(n, W, 10 * s + seed, dtype) for s, n in enumerate(lens)]
    outs, done = [[] for _ in lens], [0] * len(lens)
    portions = portions or [[n] for n in lens]
    turn = 0
    while any(d < n for d, n in zip(done, lens)):
        todo = []
        for s, n in enumerate(lens):
            if done[s] < n:
                p = portions[s]
                todo.append((s, min(p[min(turn, len(p) - 1)], n - done[s])))
        todo.sort(key=lambda e: e[1] == 1)
        y = torch.cat([torch.cat([t[done[s]:done[s] + n] for t in data[s]], 1) for s, n in todo]).to(device, dtype)
        step = make_step([(done[s], n) for s, n in todo], [tables[s] for s, _ in todo], bt, device)
        out, r = ops.gated_recurrence(y, W, state, bt, step).float().cpu(), 0
        for s, n in todo:
            outs[s].append(out[r:r + n])
            r, done[s] = r + n, done[s] + n
        turn += 1
    other = layout.view(cache, 0)
    assert bool((other == 7).all())
    for s, n in enumerate(lens):
        z, u, gg = data[s]
        S = oracle.recurrence(z.double(), u.double(), torch.zeros(W, dtype=torch.float64))
        yield torch.cat(outs[s]), S * (gg * oracle.sigmoid(gg)).double(), S, tables[s], state


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("W,bt", [(8, 16), (56, 16), (136, 5), (320, 32), (64, 1)])
def test_recurrence_portions_and_states(device, dtype, W, bt):
    lens = [1, 2, 16, 17, 127, 128, 129, 300]
    ways = {"whole": None, "single": [[1]] * 8, "mixed": [[1], [2], [3, 13], [5], [100, 1, 1, 40], [1, 127], [64], [129, 1, 2, 64, 31]]}
    for seed, portions in enumerate(ways.values()):
        for got, want, S, table, state in run_recurrence(W, lens, bt, device, dtype, portions, seed):
            close(got, want, dtype, scale=max(1.0, float(want.abs().max())))
            for b, blk in enumerate(table):              # every block keeps the state after its last token
                close(state[blk], S[min((b + 1) * bt, S.shape[0]) - 1], torch.float32, scale=40)
    if device == "cuda":
        native.check_err_flag("cuda")


@pytest.mark.parametrize("device,dtype", PLACES)
def test_recurrence_long_memory_and_wide_rows(device, dtype):
    for W, n, portions in ((40, 1500, [[1300, 1]]), (1000, 520, [[257]])) if device == "cuda" else ((40, 700, [[600, 1]]),):
        (got, want, _, _, _), = run_recurrence(W, [n], 16, device, dtype, portions, 3)
        close(got, want, dtype, scale=max(1.0, float(want.abs().max())))


@pytest.mark.parametrize("device,dtype", PLACES)
def test_recurrence_many_sequences(device, dtype):
    """More sequences than fit the narrow channel tiles' grid: the other tile width."""
    W, lens = 640, [20 + s for s in range(32)]
    for got, want, *_ in run_recurrence(W, lens if device == "cuda" else lens[:3], 16, device, dtype, None, 1):
        close(got, want, dtype, scale=max(1.0, float(want.abs().max())))


@pytest.mark.gpu
def test_recurrence_padding_rows_and_bad_blocks():
    W, bt = 24, 16
    layout = RecordLayout(torch.bfloat16)
    at = layout.add((W,), torch.float32)
    cache = torch.zeros(4, layout.record, dtype=torch.bfloat16, device="cuda")
    state = layout.view(cache, at)
    y = rand(0, 3, 3 * W).cuda().bfloat16()
    step = make_step([(0, 1), (0, 1), (0, 1)], [[2], [0], [1]], bt, "cuda")
    step.kv_lens[1], step.slots[1] = 0, -1                                  # a padding row of a captured decode step
    out = ops.gated_recurrence(y, W, state, bt, step)
    assert not out[1].any() and not state[0].any() and out[0].any() and state[2].any()
    native.clear_err_flag("cuda")
    bad = make_step([(0, 1)], [[4]], bt, "cuda")             # a block id outside the cache: recorded and skipped
    ops.gated_recurrence(y[:1], W, state, bt, bad)
    with pytest.raises(RuntimeError):
        native.check_err_flag("cuda")
    assert not state[[0, 3]].any()


# ------------------------------------------------------------------------------------------------ latents
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,dim,rot,rank,base", [(3, 16, 8, 40, 900.0), (2, 10, 6, 22, 70.0), (1, 8, 2, 3, 1e6), (5, 24, 64, 520, 5000.0),
                                                 (24, 128, 64, 512, 10000.0)])
def test_latent_norm_rotation_and_append(device, dtype, H, dim, rot, rank, base):
    bt, blocks, eps = 16, 5, 0.05
    d, r, k = up8(dim), up8(rot), up8(rank)
    positions, slots = [0, 1, 17, 63, 64, 399, 5], [3, 16, 79, 0, 40, 41, -1]          # the last row is padding: not written
    T = len(positions)
    q, kv, w = rand(0, T, H, dim + rot), rand(1, T, rank + rot) * 3, rand(2, rank)
    qp = torch.cat([pad(q[..., :dim], d), pad(q[..., dim:], r)], -1)
    kvp = torch.cat([pad(kv[:, :rank], k), pad(kv[:, rank:], r)], -1)
    rows = torch.cat([torch.full((T, 8), 9.0), qp.reshape(T, -1), kvp, torch.full((T, 16), 9.0)], 1).to(device, dtype)   # packed projections
    dq = rows[:, 8:8 + H * (d + r)].unflatten(1, (H, -1))
    dkv = rows[:, 8 + H * (d + r):8 + H * (d + r) + k + r]
    layout = RecordLayout(dtype)
    layout.add((24,), torch.float32)
    at = layout.add((bt, k + r))
    cache = torch.full((blocks, layout.record), 7.0, dtype=dtype, device=device)
    panel = layout.view(cache, at)
    i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)  # noqa: E731
    step = SimpleNamespace(positions=i32(positions), slots=i32(slots))
    table = ref.build_cos_sin_cache(rot, 400, base, None, device)
    norm = ops.NormParams(pad(w, k).to(device, dtype), None, rank, eps, rms=True)
    qfull = ops.latent_append(dq, d, dkv, norm, step, table, panel, bt)
    want = torch.full(panel.shape, 7.0)
    for t, (p, s) in enumerate(zip(positions, slots)):
        close(qfull[t, :, k:k + rot], oracle.rotate(q[t, :, dim:], p, base), dtype)
        assert not qfull[t, :, k + rot:].any()
        if s >= 0:
            c = oracle.group_norm(kv[t, :rank], w, 1, eps)
            want[s // bt, s % bt] = torch.cat([pad(c, k), pad(oracle.rotate(kv[t, rank:], p, base), r)])
    close(panel, want, dtype)
    assert bool((layout.view(cache, 0).view(dtype) == 7).all())
    # latents of another layer: the queries turn, nothing is appended
    before = cache.clone()
    again = ops.latent_append(dq, d, None, None, step, table, panel, bt)
    assert torch.equal(again[..., k:], qfull[..., k:]) and torch.equal(cache, before)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("B,M,N,K", [(3, 5, 24, 40), (1, 1, 8, 8), (16, 70, 72, 136), (2, 300, 512, 128)])
def test_batched_product(device, dtype, B, M, N, K):
    a, w = rand(0, M, B, K + 8), rand(1, B, N, K)
    out = torch.zeros(M, B, N + 16, dtype=dtype, device=device)
    ops.bmm(a.to(device, dtype)[..., :K].transpose(0, 1), w.to(device, dtype), out[..., 8:8 + N].transpose(0, 1))
    want = torch.einsum("mbk,bnk->mbn", a[..., :K].double(), w.double())
    close(out[..., 8:8 + N], want, dtype, scale=float(want.abs().max()))
    assert not out[..., :8].any() and not out[..., 8 + N:].any()
    wide = (rand(2, M, 16 + B * N) * 4).to(device, dtype)              # the gate is a column range of wider rows
    gate = wide[:, 16:].unflatten(1, (B, N))
    ops.bmm(a.to(device, dtype)[..., :K].transpose(0, 1), w.to(device, dtype), out[..., 8:8 + N].transpose(0, 1), gate.transpose(0, 1))
    want = want * oracle.sigmoid(gate.double().cpu())
    close(out[..., 8:8 + N], want, dtype, scale=float(want.abs().max()))


def latent_case(G, rank, rot, window, lens, bt, device, dtype, seed=0):
    """Sequences of (cached, new) tokens in shuffled blocks. Every query points at one key (its own, the last inside and the
    first outside the window, page and tile borders, the first ones, a random one) with a score that stands out by about
    12, so that a key wrongly seen or missed turns the output over."""
    g = torch.Generator().manual_seed(seed)
    D = rank + rot
    scale = D ** -0.5 * 1.3
    lens = sorted(lens, key=lambda e: e[1] == 1)         # multi-token sequences first
    nblk = [(p + n + bt - 1) // bt for p, n in lens]
    ids = torch.randperm(sum(nblk) + 3, generator=g).tolist()
    layout = RecordLayout(dtype)
    layout.add((5,), torch.float32)
    at = layout.add((bt, D))
    cache = torch.randn(len(ids), layout.record, generator=g).mul_(3).to(dtype).to(device)    # stale values everywhere
    panel = layout.view(cache, at)
    tables, qs, want, k = [], [], [], 0
    for s, (past, n) in enumerate(lens):
        T = past + n
        kv = torch.randn(T, D, generator=g).to(dtype).float()
        q = torch.randn(T, G, D, generator=g) * 0.3
        for i in range(T):
            for h in range(G):
                edges = [i, i - window + 1, i - window, i // bt * bt - 1, i // 64 * 64, i // 64 * 64 - 1, 0, 1,
                         int(torch.randint(0, i + 1, (1,), generator=g))]
                j = edges[(i + 5 * h) % len(edges)]
                if 0 <= j <= i:
                    q[i, h] = kv[j] * (12.0 / (scale * float(kv[j] @ kv[j])))
        q = q.to(dtype).float()
        want.append(torch.stack([oracle.attend(q[:, h], kv, kv[:, :rank], scale, window or None) for h in range(G)], 1)[past:])
        blk = ids[k:k + nblk[s]]
        k += nblk[s]
        tables.append(blk)
        for t in range(T):
            panel[blk[t // bt], t % bt] = kv[t].to(device, dtype)
        qs.append(q[past:])
    got = ops.latent_attention(torch.cat(qs).to(device, dtype).contiguous(), panel, rank, bt, make_step(lens, tables, bt, device), scale, window)
    return got, torch.cat(want)


LENS = [(0, 1), (0, 150), (63, 2), (64, 1), (130, 70), (127, 1), (200, 3), (15, 17), (255, 1), (31, 33)]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("G,rank,rot,window,bt", [
    (4, 32, 16, 40, 16), (6, 96, 32, 63, 16), (3, 24, 8, 64, 8), (1, 64, 64, 65, 32), (5, 136, 8, 1, 16), (24, 256, 64, 33, 16),
    (2, 264, 64, 128, 64), (3, 512, 64, 100, 16), (7, 40, 8, 0, 16), (2, 520, 64, 17, 16), (4, 48, 16, 30, 5), (130, 64, 16, 20, 16),
    (2, 8, 8, 1000, 16), (12, 448, 128, 129, 128)])
def test_latent_window_attention(device, dtype, G, rank, rot, window, bt):
    lens = LENS if device == "cuda" and G < 100 else [LENS[0], LENS[3], LENS[5], LENS[6], LENS[7]] + ([] if G > 20 else [LENS[4]])
    got, want = latent_case(G, rank, rot, window, lens, bt, device, dtype)
    close(got, want, dtype, scale=4 if dtype == torch.bfloat16 else None)
    if device == "cuda":
        native.check_err_flag("cuda")


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("window", [0, 300, 700])
def test_latent_attention_far_keys(device, dtype, window):
    """Hundreds of keys, a single one of which matters; long enough for several split ranges of the decode kernel."""
    for lens in ([(900, 1), (640, 1), (1, 1)], [(700, 130), (3, 2), (1023, 1)]) if device == "cuda" else ([(640, 1), (1, 2)],):
        got, want = latent_case(4, 64, 16, window, lens, 16, device, dtype, seed=3)
        close(got, want, dtype, scale=4 if dtype == torch.bfloat16 else None)


# ------------------------------------------------------------------------------------------------ the oracle's equations
def test_absorbed_form_equals_the_plain_one():
    """W_uk on the query's side and W_uv behind the weighted latents give the attention over expanded keys and values."""
    H, dim, rot, vdim, rank, T, W = 3, 10, 6, 12, 22, 40, 30
    m = {"heads": H, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": 0.3, "rot": {"base": 50.0, "dims": rot},
         "mask": {"size": 9}}
    w = {"q": rand(0, H * (dim + rot), W), "uk": rand(1, H * dim, rank), "uv": rand(2, H * vdim, rank), "g": rand(3, H * vdim, W),
         "o": torch.eye(H * vdim)}
    w = {k: t.double() for k, t in w.items()}
    h, c, r = rand(4, T, W).double() * 0.2, rand(5, T, rank).double() * 0.3, rand(6, T, rot).double()
    want = oracle.latent_attention(h, m, w, "", c, r)
    q = (h @ w["q"].t()).view(T, H, dim + rot)
    heads = []
    for a in range(H):
        qr = torch.stack([oracle.rotate(q[p, a, dim:], p, 50.0) for p in range(T)])
        ql = q[:, a, :dim] @ w["uk"].view(H, dim, rank)[a]
        o = oracle.attend(torch.cat([ql, qr], 1), torch.cat([c, r], 1), c, 0.3, 9)
        heads.append(o @ w["uv"].view(H, vdim, rank)[a].t())
    assert float((torch.cat(heads, 1) * oracle.sigmoid(h @ w["g"].t()) - want).abs().max()) < 1e-9


def test_rotation_keeps_products_of_equal_distance():
    a, b = rand(0, 8).double(), rand(1, 8).double()
    p = [float(oracle.rotate(a, i, 30.0) @ oracle.rotate(b, i - 4, 30.0)) for i in (4, 9, 200)]
    assert max(p) - min(p) < 1e-9 and abs(p[0] - float(a @ b)) > 1e-3 and math.isfinite(p[0])
