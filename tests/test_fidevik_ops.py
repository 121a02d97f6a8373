"""The mechanisms of the Fidevik family one by one: the ops (plain statements on the CPU, kernels on the GPU) against the
plain equations of fidevik_oracle."""
from types import SimpleNamespace

import pytest
import torch

import fidevik_oracle as oracle
from decoder_helpers import PLACES, TOL, close, make_step, pad, rand, up8
from ksanallm_b200.models.common import RecordLayout
from ksanallm_b200.models.moe import expert_outputs
from ksanallm_b200.models.stream import rerotate_panel
from ksanallm_b200.ops import dispatch as ops
from ksanallm_b200.ops import native
from ksanallm_b200.ops import reference as ref


# ------------------------------------------------------------------------------------------------ norms and units
def layer_norm_params(H, device, dtype, seed, eps=0.02):
    w, b = rand(seed, H) + 1, rand(seed + 1, H)
    n = ops.NormParams(pad(w, up8(H)).to(device, dtype), pad(b, up8(H)).to(device, dtype), H, eps)
    return n, lambda x: oracle.layer_norm(x, w.double(), b.double(), eps)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H", [8, 70, 256, 2050, 9000])
def test_opening_of_a_pass(device, dtype, H):
    """Stream + embedding output + step vector and the layer norm of the sum, alone and behind a sublayer's addition."""
    HP, M = up8(H), 5
    x, first, y, vec = rand(0, M, H) * 3 + 1, rand(1, M, H) * 2, rand(2, M, H), rand(3, H)
    norm, plain = layer_norm_params(H, device, dtype, 4)
    xd, fd, yd, vd = (pad(t, HP).to(device) for t in (x, first, y, vec))
    yd, vd = yd.to(dtype), vd.to(dtype)
    for add in (None, fd):
        want = x.double() + vec.double() + (0 if add is None else first.double())
        base = xd.clone()
        out, z = ops.stream_enter(base, add, vd, norm, dtype, inplace=False)
        assert out.data_ptr() != base.data_ptr() and torch.equal(base, xd) and z.dtype == dtype
        close(out[:, :H], want, torch.float32)
        close(z[:, :H], plain(want), dtype)
        assert not out[:, H:].any() and not z[:, H:].any()
        out, _ = ops.stream_enter(base, add, vd, norm, dtype)
        assert out.data_ptr() == base.data_ptr()
        out, z = ops.stream_add(xd.clone(), yd, None, None, norm, add=add, vec=vd)
        close(out[:, :H], want + y.double(), torch.float32)
        close(z[:, :H], plain(want + y.double()), dtype)
        out, z = ops.stream_add(xd.clone(), yd, None, None, None, add=add, vec=vd)
        assert z is None
        close(out[:, :H], want + y.double(), torch.float32)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("scale", [1.0, 0.31, 7.0])
def test_scaled_final_norm(device, dtype, scale):
    H, rows = 70, [3, 0, 3]
    x = rand(0, 5, H) * 2
    norm, plain = layer_norm_params(H, device, dtype, 1)
    got = ops.stream_norm(pad(x, up8(H)).to(device), norm, dtype, rows=torch.tensor(rows, dtype=torch.int32, device=device), scale=scale)
    close(got[:, :H], plain(x.double())[rows] * scale, dtype)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("kind,act", [("silu", oracle.silu), ("gelu", oracle.gelu)])
def test_gated_units(device, dtype, kind, act):
    x = torch.cat([rand(0, 40, 48) * 3, torch.tensor([0.0, -0.0, 1e-3, -1e-3, -3.0, -6.0, 12.0, -90.0] * 6).view(1, 48)]).to(dtype)
    close(ops.act_mul(x.to(device), kind), act(x[:, :24].double()) * x[:, 24:].double(), dtype)


# ------------------------------------------------------------------------------------------------ experts
def well_apart(E, T, seed, count, keep, top):
    """Logits and corrections whose choices do not hinge on rounding: scores a good step apart, in another order for every token
    (the corrections put many choice scores below zero)."""
    g = torch.Generator().manual_seed(seed)
    corr = torch.randint(-6, 3, (E,), generator=g).float() * 0.25
    rows, chosen = [], []
    while len(rows) < T:
        z = torch.randn(E, generator=g) * 2
        choice = (oracle.sigmoid(z) + corr).double()
        size = E // count
        groups = choice.view(count, size).sort(-1).values[:, -2:].sum(-1)
        order = groups.sort().values
        if keep < count and float(order[-keep] - order[-keep - 1]) < 1e-4:
            continue
        w = oracle.choose(z.double(), corr.double(), top, count, keep)
        kept = set(groups.topk(keep).indices.tolist())
        rest = [float(choice[e]) for e in range(E) if e // size in kept and e not in w]
        if rest and min(float(choice[e]) for e in w) - max(rest) < 1e-4:
            continue
        rows.append(z)
        chosen.append(w)
    return torch.stack(rows), corr, chosen


ROUTERS = [(14, 3, 2, 1), (12, 4, 4, 2), (9, 2, 3, 3), (1, 1, 1, 1), (4, 2, 4, 3), (64, 8, 8, 3), (80, 12, 40, 9), (512, 20, 64, 4), (33, 33, 1, 1),
           (40, 5, 20, 3)]


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("E,top,count,keep", ROUTERS)
def test_choice_of_experts(device, E, top, count, keep):
    T = 37
    z, corr, want = well_apart(E, T, E + top, count, keep, top)
    gate = rand(5, T, 1) * 3
    logits = torch.cat([z, gate, torch.full((T, 4), 50.0)], 1).to(device)           # columns behind the experts' do not count
    kw = dict(scoring="sigmoid", renorm=False, bias=corr.to(device), n_group=count, topk_group=keep, E=E)
    ids, w = ops.moe_route(logits, top, gate_col=E, **kw)
    assert ids.dtype == torch.int32 and tuple(w.shape) == (T, top + 1)
    close(w[:, top:], oracle.sigmoid(gate), torch.float32)
    ids2, w2 = ops.moe_route(logits, top, **kw)
    assert torch.equal(ids, ids2) and torch.equal(w2, w[:, :top])
    for t in range(T):
        got = {int(e): float(v) for e, v in zip(ids[t].cpu(), w[t, :top].cpu())}
        assert got.keys() == want[t].keys()
        for e, v in want[t].items():
            assert abs(got[e] - float(v)) < 1e-5                                     # the score, without the correction


def test_choice_notices():
    """What the routing cases tell apart: the groups, the corrections in the choice, and their absence from the weights."""
    z, corr, want = well_apart(12, 200, 3, 4, 2, 4)
    other = [oracle.choose(r.double(), corr.double(), 4, 1, 1) for r in z]
    plain = [oracle.choose(r.double(), corr.double() * 0, 4, 4, 2) for r in z]
    assert sum(a.keys() != b.keys() for a, b in zip(want, other)) > 100
    assert sum(a.keys() != b.keys() for a, b in zip(want, plain)) > 100
    negative = sum(float(oracle.sigmoid(r)[e] + corr[e]) < 0 for r, c in zip(z, want) for e in c)
    assert negative > 20                                                              # experts chosen with a negative score


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,K,shared", [(8, 1, False), (70, 3, True), (256, 8, True), (2050, 2, False), (4104, 5, True)])
def test_weighted_sum_of_expert_rows(device, dtype, H, K, shared):
    HP, T, cap = up8(H), 6, 60
    g = torch.Generator().manual_seed(H)
    x, y, w, s = rand(0, T, H), rand(1, cap, H), rand(2, T, K + shared).abs(), rand(3, T, H)
    dst = torch.randperm(cap, generator=g)[:T * K].view(T, K).to(torch.int32)
    dst[1, 0] = -1                                                                    # an expert that lives elsewhere
    want = x.double()
    for t in range(T):
        for k in range(K):
            if dst[t, k] >= 0:
                want[t] += w[t, k].double() * y[dst[t, k]].double()
        if shared:
            want[t] += w[t, K].double() * s[t].double()
    yd = pad(y, HP).to(device, dtype).clone()
    yd[[r for r in range(cap) if r not in dst.flatten().tolist()]] = float("nan")     # rows that nobody chose are not read
    e = ops.ExpertSum(yd, dst.to(device), w.to(device), pad(s, HP).to(device, dtype) if shared else None)
    norm, plain = layer_norm_params(H, device, dtype, 7)
    out, z = ops.stream_add(pad(x, HP).to(device).clone(), e, None, None, norm)
    close(out[:, :H], want, torch.float32)
    close(z[:, :H], plain(want), dtype)
    out, z = ops.stream_add(pad(x, HP).to(device).clone(), e, None, None, None, vec=pad(rand(9, H), HP).to(device, dtype))
    close(out[:, :H], want + rand(9, H).double(), torch.float32)
    if device == "cuda":
        native.check_err_flag("cuda")


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("E,K,W,I,T", [(1, 1, 64, 8, 3), (5, 2, 72, 24, 1), (12, 4, 264, 104, 150), (40, 6, 128, 136, 300), (3, 3, 64, 40, 129)])
def test_expert_outputs(device, dtype, E, K, W, I, T):
    """Rows of experts with very different weights, several tiles of some experts, one that nobody chooses."""
    g = torch.Generator().manual_seed(E)
    x = rand(0, T, W)
    w13 = rand(1, E, 2 * I, W) * W ** -0.5 * torch.linspace(0.5, 2, E).view(E, 1, 1)
    w2 = rand(2, E, W, I) * I ** -0.5
    w13, w2 = w13.bfloat16().float(), w2.bfloat16().float()
    ids = torch.stack([torch.randperm(max(K, E - 1), generator=g)[:K] for _ in range(T)]).to(torch.int32)
    y, dst = expert_outputs(x.to(device, dtype), ids.to(device), w13.reshape(-1, W).to(device, dtype), w2.reshape(-1, I).to(device, dtype), I)
    assert tuple(dst.shape) == (T, K)
    got = y[dst.long().flatten()].view(T, K, W)
    want = torch.zeros(T, K, W, dtype=torch.float64)
    for e in range(E):
        w = {"gate": w13[e, :I].double(), "up": w13[e, I:].double(), "down": w2[e].double()}
        want[ids == e] = oracle.gated_unit(x.double(), w, "", oracle.silu)[(ids == e).nonzero()[:, 0]]
    close(got, want, dtype)


# ------------------------------------------------------------------------------------------------ queries, keys, latents
def i32(t, device):
    return torch.tensor(t, dtype=torch.int32, device=device)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,G,dim,vdim,rot,base", [(4, 2, 16, 24, 16, 900.0), (3, 1, 10, 6, 6, 70.0), (2, 2, 20, 8, 14, 1e6), (6, 3, 64, 64, 0, 1.0),
                                                   (1, 1, 2, 1, 2, 10.0), (32, 8, 128, 128, 64, 10000.0), (5, 5, 200, 136, 36, 500.0)])
def test_query_key_norm_rotation_and_append(device, dtype, H, G, dim, vdim, rot, base):
    bt, blocks, eps, D, DV = 16, 5, 0.05, up8(dim), up8(vdim)
    positions, slots = [0, 1, 17, 63, 64, 399, 5], [3, 16, 79, 0, 40, 41, -1]          # the last row is padding: not written
    T = len(positions)
    q, k, v = rand(0, T, H, dim) * 2, rand(1, T, G, dim) * 0.3, rand(2, T, G, vdim)
    q[0, 0] *= 30                                        # one head that dominates the row's norm
    q, k = q.bfloat16().float(), k.bfloat16().float()
    qw, kw = rand(3, H, dim), rand(4, G, dim)
    rows = torch.cat([pad(q, D).flatten(1), pad(k, D).flatten(1), pad(v, DV).flatten(1)], 1)
    layout = RecordLayout(dtype)
    layout.add((24,))
    ki, vi = layout.add((G, bt, D)), layout.add((G, bt, DV))
    norms = [ops.NormParams(pad(w, D).flatten().to(device, dtype), None, w.numel(), eps, rms=True) for w in (qw, kw)]
    table = ref.build_cos_sin_cache(rot, 400, base, None, device) if rot else None
    step = SimpleNamespace(positions=i32(positions, device), slots=i32(slots, device))
    want_q = oracle.rms_norm(q.flatten(1), qw.flatten(), eps).view(T, H, dim)
    want_k = oracle.rms_norm(k.flatten(1), kw.flatten(), eps).view(T, G, dim)
    want_q, want_k = (torch.stack([oracle.rotate(t[p], positions[p], rot, base) for p in range(T)]) for t in (want_q, want_k))
    full = torch.stack([q.flatten(1).pow(2).sum(1), k.flatten(1).pow(2).sum(1)], 1).to(device)
    for sums in (None, full):                            # the sums of squares may come from elsewhere
        cache = torch.full((blocks, layout.record), 7.0, dtype=dtype, device=device)
        kp, vp = layout.view(cache, ki), layout.view(cache, vi)
        qkv = rows.to(device, dtype).clone()
        ops.qkv_norm_rope_append(qkv, step, table, *norms, kp, vp, bt, H, G, rot, sums)
        got_q = qkv[:, :H * D].unflatten(1, (H, D))
        close(got_q[..., :dim], want_q, dtype)
        assert not got_q[..., dim:].any()
        wk, wv = torch.full(kp.shape, 7.0), torch.full(vp.shape, 7.0)
        for t, s in enumerate(slots):
            if s >= 0:
                wk[s // bt, :, s % bt], wv[s // bt, :, s % bt] = pad(want_k[t], D), pad(v[t], DV)
        close(kp, wk, dtype)
        close(vp, wv, dtype)
        assert bool((layout.view(cache, 0) == 7).all())


@pytest.mark.parametrize("device,dtype", PLACES)
def test_moved_keys_are_turned(device, dtype):
    """A copied block's keys turn by the position delta, in either direction; the other dimensions and blocks stay."""
    rot, D, bt, base = 6, 16, 8, 70.0
    table = ref.build_cos_sin_cache(rot, 300, base, None, device)
    layout = RecordLayout(dtype)
    layout.add((8,))
    at = layout.add((2, bt, D))
    cache = torch.zeros(4, layout.record, dtype=dtype, device=device)
    panel = layout.view(cache, at)
    raw = rand(0, 2, bt, D)
    panel[1] = oracle.rotate(raw, 40, rot, base).to(device, dtype)
    panel[3] = panel[1]
    panel[2] = panel[1]
    rerotate_panel(panel, torch.tensor([[0, 1, 25], [0, 3, -33]]), table, interleaved=True)
    close(panel[1], oracle.rotate(raw, 65, rot, base), dtype)
    close(panel[3], oracle.rotate(raw, 7, rot, base), dtype)
    close(panel[2], oracle.rotate(raw, 40, rot, base), dtype)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("q_rank,kv_rank", [(24, 40), (13, 22), (1, 3), (136, 8), (1536, 512), (2304, 2500)])
def test_latent_norms_and_append(device, dtype, q_rank, kv_rank):
    bt, blocks, eps, qp, kp = 16, 5, 0.05, up8(q_rank), up8(kv_rank)
    slots = [3, 16, 79, 0, 40, 41, -1]
    T = len(slots)
    q, kv, qw, kw = rand(0, T, q_rank) * 3, rand(1, T, kv_rank) * 0.2, rand(2, q_rank), rand(3, kv_rank)
    rows = torch.cat([torch.full((T, 8), 9.0), pad(q, qp), pad(kv, kp), torch.full((T, 16), 9.0)], 1).to(device, dtype)
    layout = RecordLayout(dtype)
    layout.add((5,), torch.float32)
    at = layout.add((bt, kp))
    cache = torch.full((blocks, layout.record), 7.0, dtype=dtype, device=device)
    norms = [ops.NormParams(pad(w, up8(w.numel())).to(device, dtype), None, w.numel(), eps, rms=True) for w in (qw, kw)]
    panel = layout.view(cache, at)
    got = ops.latent_norms(rows[:, 8:8 + qp], rows[:, 8 + qp:8 + qp + kp], *norms, SimpleNamespace(slots=i32(slots, device)), panel, bt)
    close(got[:, :q_rank], oracle.rms_norm(q, qw, eps), dtype)
    assert not got[:, q_rank:].any()
    want = torch.full(panel.shape, 7.0)
    for t, s in enumerate(slots):
        if s >= 0:
            want[s // bt, s % bt] = pad(oracle.rms_norm(kv[t], kw, eps), kp)
    close(panel, want, dtype)
    assert bool((layout.view(cache, 0).view(dtype) == 7).all())


# ------------------------------------------------------------------------------------------------ attention
def pointed(g, k, H, i, h, bt, scale, height):
    """A query at position i that points at one key of k [T, D]: its own, a page or tile border, one of the first, any. Its score
    is ``height``."""
    edges = [i, i // bt * bt - 1, i // bt * bt, i // 64 * 64, i // 64 * 64 - 1, 0, 1, i // 128 * 128 - 1,
             int(torch.randint(0, i + 1, (1,), generator=g))]
    j = edges[(i + 5 * h) % len(edges)]
    if not 0 <= j <= i:
        j = i
    return k[j] * (height / (scale * float(k[j] @ k[j])))


def paged(data, lens, bt, layout, at, device, dtype, g):
    """Scatters per-sequence rows into shuffled blocks of a cache full of stale values: (panels, block ids per sequence)."""
    nblk = [(p + n + bt - 1) // bt for p, n in lens]
    ids = torch.randperm(sum(nblk) + 3, generator=g).tolist()
    cache = torch.randn(len(ids), layout.record, generator=g).mul_(3).to(dtype).to(device)
    panels, tables, k = [layout.view(cache, i) for i in at], [], 0
    for s, n in enumerate(nblk):
        tables.append(ids[k:k + n])
        k += n
        for panel, rows in zip(panels, data[s]):
            for t in range(rows.shape[0]):
                panel[(tables[s][t // bt], t % bt) if panel.dim() == 3 else (tables[s][t // bt], slice(None), t % bt)] = rows[t].to(device, dtype)
    return panels, tables


LENS = [(0, 1), (0, 150), (63, 2), (64, 1), (130, 70), (127, 1), (200, 3), (15, 17), (255, 1), (31, 33)]


def latent_case(G, rank, lens, bt, device, dtype, seed=0):
    """Queries that point at single keys; sinks from negligible over equal to the pointed score to overwhelming, head by head;
    gates on both sides of zero."""
    g = torch.Generator().manual_seed(seed)
    scale = rank ** -0.5 * 1.3
    lens = sorted(lens, key=lambda e: e[1] == 1)
    sinks = torch.tensor([-20.0, 12.0, 11.0, 13.5, 2.0, 30.0])[torch.arange(G) % 6]
    data, qs, gates, want = [], [], [], []
    for past, n in lens:
        c = torch.randn(past + n, rank, generator=g).to(dtype).float()
        q = torch.randn(past + n, G, rank, generator=g) * 0.3
        for i in range(past + n):
            for h in range(G):
                if rank >= 8:
                    q[i, h] = pointed(g, c, G, i, h, bt, scale, 12.0)
        q, gate = q.to(dtype).float(), (torch.randn(past + n, G, generator=g) * 2).to(dtype).float()
        heads = [oracle.attend(q[:, h], c, c, scale, sinks[h]) * oracle.sigmoid(gate[:, h:h + 1]) for h in range(G)]
        data.append((pad(c, up8(rank)),))
        qs.append(q[past:])
        gates.append(gate[past:])
        want.append(torch.stack(heads, 1)[past:])
    layout = RecordLayout(dtype)
    layout.add((5,), torch.float32)
    (panel,), tables = paged(data, lens, bt, layout, [layout.add((bt, up8(rank)))], device, dtype, g)
    q = pad(torch.cat(qs), up8(rank)).to(device, dtype).contiguous()
    wide = pad(torch.cat(gates), G + 11).to(device, dtype)                       # the gate is a column range of wider rows
    got = ops.latent_attention(q, panel, up8(rank), bt, make_step(lens, tables, bt, device), scale, 0, sinks.to(device), wide[:, :G])
    return got[..., :rank], torch.cat(want)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("G,rank,bt", [(4, 32, 16), (6, 96, 16), (3, 24, 8), (1, 64, 32), (5, 136, 16), (24, 256, 16), (2, 264, 64), (3, 512, 16),
                                       (7, 40, 16), (2, 520, 16), (4, 48, 5), (130, 64, 16), (2, 200, 16), (12, 440, 128), (3, 330, 16)])
def test_latent_attention_with_sinks_and_gates(device, dtype, G, rank, bt):
    lens = LENS if device == "cuda" and G < 100 else [LENS[0], LENS[3], LENS[5], LENS[6], LENS[7]] + ([] if G > 20 else [LENS[4]])
    got, want = latent_case(G, rank, lens, bt, device, dtype)
    close(got, want, dtype, scale=4 if dtype == torch.bfloat16 else None)
    if device == "cuda":
        native.check_err_flag("cuda")


@pytest.mark.parametrize("device,dtype", PLACES)
def test_latent_attention_far_keys(device, dtype):
    """Hundreds of keys, a single one of which matters; long enough for several split ranges of the decode kernel, whose parts
    must meet one sink and one gate."""
    for lens in ([(900, 1), (640, 1), (1, 1)], [(700, 130), (3, 2), (1023, 1)]) if device == "cuda" else ([(640, 1), (1, 2)],):
        got, want = latent_case(6, 64, lens, 16, device, dtype, seed=3)
        close(got, want, dtype, scale=4 if dtype == torch.bfloat16 else None)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("window", [1, 64, 100])
def test_sinks_with_a_window(device, dtype, window):
    """The same kernels with a sliding window: uniform keys, so that a row's weight on its values is n e^s / (n e^s + e^sink)."""
    G, rank, bt, lens = 3, 32, 16, [(0, 150), (64, 3), (130, 1)]
    sinks = torch.tensor([0.0, 3.0, 6.0])
    layout = RecordLayout(dtype)
    rows = [(torch.ones(p + n, rank),) for p, n in lens]
    (panel,), tables = paged(rows, lens, bt, layout, [layout.add((bt, rank))], device, dtype, torch.Generator().manual_seed(1))
    q = torch.full((154, G, rank), 1.0 / rank, dtype=dtype, device=device)
    got = ops.latent_attention(q, panel, rank, bt, make_step(lens, tables, bt, device), 2.0, window, sinks.to(device))
    pos = torch.cat([torch.arange(p, p + n) for p, n in lens])
    n = torch.minimum(pos + 1, torch.tensor(window)).double().unsqueeze(1)
    e2 = torch.exp(torch.tensor(2.0, dtype=torch.float64))
    close(got, (n * e2 / (n * e2 + torch.exp(sinks.double()))).unsqueeze(-1).expand(-1, -1, rank), dtype)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,G,D,DV,bt", [(4, 2, 16, 24, 16), (6, 1, 40, 8, 8), (8, 8, 64, 64, 16), (34, 2, 128, 56, 32), (3, 3, 200, 136, 16)])
def test_grouped_attention_over_all_keys(device, dtype, H, G, D, DV, bt):
    g = torch.Generator().manual_seed(D)
    scale = D ** -0.5
    lens = sorted(LENS if device == "cuda" else LENS[:1] + LENS[2:8], key=lambda e: e[1] == 1) + ([(700, 1)] if device == "cuda" else [])
    data, qs, want = [], [], []
    for past, n in lens:
        k, v = (torch.randn(past + n, G, m, generator=g).to(dtype).float() for m in (D, DV))
        q = torch.stack([torch.stack([pointed(g, k[:, h // (H // G)], H, i, h, bt, scale, 12.0) for h in range(H)]) for i in range(past, past + n)])
        q = torch.cat([torch.zeros(past, H, D), q.to(dtype).float()])
        want.append(torch.cat([oracle.attend(q[:, h], k[:, h // (H // G)], v[:, h // (H // G)], scale) for h in range(H)], 1)[past:])
        data.append((k, v))
        qs.append(q[past:].flatten(1))
    layout = RecordLayout(dtype)
    layout.add((8,))
    (kp, vp), tables = paged(data, lens, bt, layout, [layout.add((G, bt, D)), layout.add((G, bt, DV))], device, dtype, g)
    qkv = pad(torch.cat(qs), H * D + G * (D + DV)).to(device, dtype)
    got = ops.panel_attention(qkv, kp, vp, bt, make_step(lens, tables, bt, device), H, G, scale)
    close(got, torch.cat(want), dtype, scale=4 if dtype == torch.bfloat16 else None)


# ------------------------------------------------------------------------------------------------ the oracle's equations
def test_absorbed_form_equals_the_plain_one():
    """W_uk on the query's side, W_uv behind the weighted latents, the gate on those instead of on the values: the same."""
    H, d, v, qr, rank, T, W, eps = 3, 10, 12, 14, 22, 40, 30, 0.01
    m = {"heads": H, "dim": d, "vdim": v, "q_rank": qr, "kv_rank": rank, "scale": 0.3}
    w = {"dq": rand(0, qr, W), "dq.norm": rand(1, qr), "uq": rand(2, H * d, qr), "dkv": rand(3, rank, W), "dkv.norm": rand(4, rank),
         "uk": rand(5, H * d, rank), "uv": rand(6, H * v, rank), "sink": rand(7, H), "g": rand(8, H, W), "o": torch.eye(H * v)}
    w = {k: t.double() for k, t in w.items()}
    h = rand(9, T, W).double() * 0.2
    c = oracle.rms_norm(h @ w["dkv"].t(), w["dkv.norm"], eps)
    q = (oracle.rms_norm(h @ w["dq"].t(), w["dq.norm"], eps) @ w["uq"].t()).view(T, H, d)
    heads = []
    for a in range(H):
        o = oracle.attend(q[:, a] @ w["uk"].view(H, d, rank)[a], c, c, 0.3, w["sink"][a]) * oracle.sigmoid(h @ w["g"][a]).unsqueeze(1)
        heads.append(o @ w["uv"].view(H, v, rank)[a].t())
    assert float((torch.cat(heads, 1) - oracle.latent_attention(h, m, w, "", eps)).abs().max()) < 1e-9


def test_a_sink_takes_its_share():
    k = torch.zeros(3, 4, dtype=torch.float64)
    v = torch.ones(3, 2, dtype=torch.float64)
    out = oracle.attend(k, k, v, 1.0, torch.tensor(0.0, dtype=torch.float64))
    assert torch.allclose(out[:, 0], torch.tensor([1 / 2, 2 / 3, 3 / 4], dtype=torch.float64)) and TOL[torch.float32] < 1e-3
