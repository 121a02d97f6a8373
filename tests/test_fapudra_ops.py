"""The mechanisms of the Fapudra family one by one: the ops (plain statements on the CPU, kernels on the GPU) against the plain
equations of fapudra_oracle."""
from types import SimpleNamespace

import pytest
import torch

import fapudra_oracle as oracle
from decoder_helpers import PLACES, TOL, close, make_step, pad, rand, up8
from ksanallm_b200.config import MlpSpec
from ksanallm_b200.models.common import RecordLayout
from ksanallm_b200.models.moe import expert_outputs
from ksanallm_b200.models.stream import distance_biases
from ksanallm_b200.ops import dispatch as ops
from ksanallm_b200.ops import native

NAN = float("nan")


def fault_free(device):
    if device == "cuda":
        native.check_err_flag("cuda")


# ------------------------------------------------------------------------------------------------ rows
@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("W", [8, 70, 256, 2050, 9000])
def test_normed_embedding(device, dtype, W):
    table, pos, g, P = rand(0, 30, W), rand(1, 17, W), 1.25, up8(W)
    ids, at = torch.tensor([0, 29, 7, 7, 3]), torch.tensor([0, 16, 2, 3, 9])
    norm = ops.NormParams(pad(torch.full((W,), g), P).to(device, dtype), None, W, 1e-3, rms=True)
    x = ops.embed_normed(ids.int().to(device), at.int().to(device), pad(table, P).to(device, dtype), pad(pos, P).to(device, dtype), 2.7, norm, 30)
    assert x.dtype == torch.float32 and not x[:, W:].any()
    close(x[:, :W], oracle.rms(table.double()[ids] * 2.7 + pos.double()[at], 1e-3) * g, torch.float32)
    fault_free(device)


PORTIONS = [[61], [2, 59], [1] * 7 + [2, 3, 8, 9, 30, 2], [17, 1, 16, 2, 25], [8, 8, 8, 1, 36]]


def step_of(parts, slots, device):
    """Step of sequences (cached, new, slot), multi-token ones first."""
    step = make_step([(p, n) for p, n, _ in parts], [[0] for _ in parts], 4096, device)
    step.state_slots = torch.tensor([s for _, _, s in parts], dtype=torch.int32, device=device)
    return step


def through(run, x_of, sizes, slot, device):
    """Rows of one sequence that arrives in portions of the given sizes."""
    out, at = [], 0
    for n in sizes:
        out.append(run(x_of(at, at + n), step_of([(at, n, slot)], None, device)).float().cpu())
        at += n
    return torch.cat(out)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("W", [8, 72, 4104])
def test_token_shift(device, dtype, W):
    h, mu = rand(0, 61, W), rand(1, W)
    want = oracle.token_shift(h.double(), mu.double())
    lay = RecordLayout(torch.float32)
    lay.add((8,))
    i = lay.add((2, W), dtype)
    state = torch.full((3, lay.record), NAN, device=device)           # whatever an earlier sequence left
    ring = lay.view(state, i)
    hd, md = h.to(device, dtype), mu.to(device, dtype)
    for slot, sizes in enumerate(PORTIONS):
        got = through(lambda x, st: ops.token_shift(x, md, ring, st), lambda a, b: hd[a:b], sizes, slot % 3, device)
        close(got, want, dtype)
    fault_free(device)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("heads,real,parts", [(1, 8, 1), (6, 16, 3), (6, 16, 1), (6, 16, 6), (3, 10, 5), (3, 10, 1), (5, 7, 7), (64, 64, 64), (32, 128, 8),
                                              (1, 1, 1), (40, 136, 4)])
def test_gated_norm(device, dtype, heads, real, parts):
    T, P = 5, up8(real)
    y, z, g, w = (rand(k, T, heads, real) * 2 for k in range(4))
    w = w[0]
    put = lambda t: pad(t, P).flatten(-2).to(device, dtype)  # noqa: E731
    plain = oracle.rms((y.double() * oracle.silu(z.double())).flatten(1).unflatten(1, (parts, -1)), 1e-2).flatten(1) * w.double().flatten()
    unpad = lambda t: t.unflatten(1, (heads, P))[..., :real].flatten(1)  # noqa: E731
    got = ops.gated_norm(put(y), put(w), 1e-2, heads, real, parts, z=put(z))
    close(unpad(got), plain, dtype, max(1.0, float(plain.abs().max())))
    assert not got.unflatten(1, (heads, P))[..., real:].any()
    wide = torch.zeros(T, heads * P + 16, device=device, dtype=dtype)
    ops.gated_norm(put(y), put(w), 1e-2, heads, real, parts, g=put(g), factor=1.4, out=wide[:, 8:8 + heads * P])
    plain = oracle.rms(y.double().flatten(1).unflatten(1, (parts, -1)), 1e-2).flatten(1) * w.double().flatten() * oracle.sigmoid(g.double()).flatten(1) * 1.4
    close(unpad(wide[:, 8:8 + heads * P]), plain, dtype, max(1.0, float(plain.abs().max())))
    assert not wide[:, :8].any() and not wide[:, 8 + heads * P:].any()


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("cap", [0.5, 24.0])
def test_softcap(device, cap):
    z = torch.cat([rand(0, 3, 100) * 40, rand(1, 3, 100) * 1e-3])
    want = cap * torch.tanh(z.double() / cap)
    close(ops.softcap(z.clone().to(device), cap), want, torch.float32, cap)
    wide = torch.zeros(6, 128, device=device)
    wide[:, :100] = z.to(device)
    close(ops.softcap(wide[:, :100], cap), want, torch.float32, cap)


# ------------------------------------------------------------------------------------------------ recurrences
def state_record(taps, channels, shape, dtype, device, slots=3):
    lay = RecordLayout(torch.float32)
    lay.add((4,))
    a, b = lay.add((taps, channels), dtype), lay.add(shape)
    state = torch.full((slots, lay.record), NAN, device=device)
    return lay.view(state, a), lay.view(state, b), state


def padded_channels(parts):
    """parts: (tensor [..., heads * real], heads) -> [..., channels] with every head padded."""
    out = []
    for t, n in parts:
        real = t.shape[-1] // n
        out.append(pad(t.unflatten(-1, (n, real)), up8(real)).flatten(-2))
    return torch.cat(out, -1)


def space_case(H, P, N, G, taps, T, seed=0, shift=0.0):
    x, B, C = rand(seed, T, H * P), rand(seed + 1, T, G * N), rand(seed + 2, T, G * N)
    dt, w, b = rand(seed + 3, T, H), rand(seed + 4, H * P + 2 * G * N, taps), rand(seed + 5, H * P + 2 * G * N) * 0.3
    A_log, D, dt_bias = rand(seed + 6, H) - 1, rand(seed + 7, H), rand(seed + 8, H) - 3 + shift          # decays from slow to moderate
    c = oracle.silu(oracle.causal_conv(torch.cat([x, B, C], 1).double(), w.double(), b.double()))
    cx, cB, cC = c.split([H * P, G * N, G * N], 1)
    step = oracle.softplus(dt.double() + dt_bias.double())
    want = torch.cat([oracle.state_space(cx[:, h * P:(h + 1) * P], cB[:, h // (H // G) * N:(h // (H // G) + 1) * N],
                                         cC[:, h // (H // G) * N:(h // (H // G) + 1) * N], step[:, h], A_log[h].double(), D[h].double())
                      for h in range(H)], 1)
    return SimpleNamespace(raw=padded_channels([(x, H), (B, G), (C, G)]), dt=pad(dt, up8(H)), want=want, A=A_log.exp(), D=D, dt_bias=dt_bias,
                           w=padded_channels([(t, n) for t, n in zip(w.t().split([H * P, G * N, G * N], 1), (H, G, G))]),
                           b=padded_channels([(t, n) for t, n in zip(b.split([H * P, G * N, G * N]), (H, G, G))]))


SPACES = [(1, 1, 1, 1, 1), (6, 16, 24, 2, 3), (3, 10, 13, 3, 2), (4, 24, 16, 4, 4), (8, 64, 128, 2, 4), (2, 72, 136, 2, 6), (5, 40, 64, 1, 3),
          (2, 33, 256, 1, 4), (2, 136, 48, 1, 4)]
# bf16 rounds the convolved inputs; everything behind them is 32-bit
LOOSE = {torch.float32: 1.0, torch.bfloat16: 2.0}


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,P,N,G,taps", SPACES)
def test_state_space(device, dtype, H, P, N, G, taps):
    k = space_case(H, P, N, G, taps, 61, H + N)
    put = lambda t: t.to(device, dtype).contiguous()  # noqa: E731
    ring, S, _ = state_record(taps, k.raw.shape[1], (H, up8(P), up8(N)), dtype, device)
    conv = ops.ShortConv(put(k.w), put(k.b), ring)
    raw, dt = put(torch.cat([k.raw, k.dt, torch.full((61, 8), NAN)], 1)), None
    C = k.raw.shape[1]
    unpad = lambda t: t.unflatten(1, (H, up8(P)))[..., :P].flatten(1)  # noqa: E731
    f32 = lambda t: t.to(device)  # noqa: E731

    def run(rows, st):
        return ops.state_space(rows[:, :C], conv, rows[:, C:], f32(k.dt_bias), f32(k.A), f32(k.D), S, G, st)

    for slot, sizes in enumerate(PORTIONS + [[1] * 61]):
        got = through(run, lambda a, b: raw[a:b], sizes, slot % 3, device)
        close(unpad(got), k.want, dtype, LOOSE[dtype] * max(1.0, float(k.want.abs().max())))
        if sizes == [61]:
            whole = S[slot % 3].clone()
    close(S[(len(PORTIONS)) % 3], whole.cpu(), dtype)               # the same state by single tokens as by one scan
    fault_free(device)


def delta_case(H, G, K, V, taps, T, seed=0, shift=0.0):
    q, kk, v = rand(seed, T, G * K), rand(seed + 1, T, G * K), rand(seed + 2, T, H * V)
    w = rand(seed + 3, 2 * G * K + H * V, taps)
    beta, decay, bias, A_log = rand(seed + 4, T, H), rand(seed + 5, T, H * K), rand(seed + 6, H * K) - 4 + shift, rand(seed + 7, H) - 1
    c = oracle.silu(oracle.causal_conv(torch.cat([q, kk, v], 1).double(), w.double()))
    cq, ck, cv = c.split([G * K, G * K, H * V], 1)
    cq, ck = oracle.unit(cq.view(T, G, K)) * K ** -0.5, oracle.unit(ck.view(T, G, K))
    step = oracle.softplus(decay.double() + bias.double()).view(T, H, K)
    g = torch.exp(-torch.exp(A_log.double())[None, :, None] * step)
    want = torch.cat([oracle.delta_rule(cq[:, h // (H // G)], ck[:, h // (H // G)], cv[:, h * V:(h + 1) * V],
                                        oracle.sigmoid(beta.double())[:, h], g[:, h]) for h in range(H)], 1)
    parts = [G * K, G * K, H * V]
    return SimpleNamespace(raw=padded_channels([(q, G), (kk, G), (v, H)]), beta=pad(beta, up8(H)), decay=padded_channels([(decay, H)]),
                           bias=padded_channels([(bias, H)]), A=A_log.exp(), want=want,
                           w=padded_channels([(t, n) for t, n in zip(w.t().split(parts, 1), (G, G, H))]))


# the last ones: more columns of states than one wave of 64 each
DELTAS = [(1, 1, 2, 1, 1), (4, 2, 16, 24, 4), (3, 3, 10, 6, 3), (2, 2, 24, 8, 2), (4, 2, 64, 64, 4), (2, 1, 128, 128, 3), (2, 1, 136, 40, 6),
          (6, 2, 40, 136, 4), (1, 1, 256, 72, 4), (80, 2, 128, 72, 4), (80, 4, 24, 128, 3)]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,G,K,V,taps", DELTAS)
def test_delta_rule(device, dtype, H, G, K, V, taps):
    k = delta_case(H, G, K, V, taps, 61, H + K)
    put = lambda t: t.to(device, dtype).contiguous()  # noqa: E731
    C = k.raw.shape[1]
    ring, S, _ = state_record(taps, C, (H, up8(V), up8(K)), dtype, device)
    conv = ops.ShortConv(put(k.w), None, ring)
    rows = put(torch.cat([k.raw, k.beta, k.decay, torch.full((61, 8), NAN)], 1))
    nb = k.beta.shape[1]
    unpad = lambda t: t.unflatten(1, (H, up8(V)))[..., :V].flatten(1)  # noqa: E731

    def run(r, st):
        return ops.delta_rule(r[:, :C], conv, r[:, C:], r[:, C + nb:C + nb + k.decay.shape[1]].contiguous(), k.bias.to(device), k.A.to(device), S, G,
                              K ** -0.5, st)

    for slot, sizes in enumerate(PORTIONS + [[1] * 61]):
        got = through(run, lambda a, b: rows[a:b], sizes, slot % 3, device)
        close(unpad(got), k.want, dtype, LOOSE[dtype] * max(1.0, float(k.want.abs().max())))
        if sizes == [61]:
            whole = S[slot % 3].clone()
    close(S[(len(PORTIONS)) % 3], whole.cpu(), dtype)
    fault_free(device)


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("shift", [0.0, 8.0, 60.0])
def test_long_prompts_and_strong_decays(device, dtype, shift):
    """Many chunks in one portion, and decays down to nothing within a token (cumulated over a chunk they are beyond fp32's range)."""
    T = 300 if device == "cuda" else 90
    k = space_case(2, 64, 128, 1, 4, T, 7, shift)
    put = lambda t: t.to(device, dtype).contiguous()  # noqa: E731
    C = k.raw.shape[1]
    ring, S, _ = state_record(4, C, (2, 64, 128), dtype, device)
    rows = put(torch.cat([k.raw, k.dt], 1))
    got = [ops.state_space(rows[a:b, :C], ops.ShortConv(put(k.w), put(k.b), ring), rows[a:b, C:], k.dt_bias.to(device), k.A.to(device),
                           k.D.to(device), S, 1, step_of([(a, b - a, 1)], None, device)).float().cpu() for a, b in ((0, T - 70), (T - 70, T))]
    close(torch.cat(got), k.want, dtype, LOOSE[dtype] * max(1.0, float(k.want.abs().max())))
    k = delta_case(2, 1, 128, 128, 4, T, 9, shift)
    C = k.raw.shape[1]
    ring, S, _ = state_record(4, C, (2, 128, 128), dtype, device)
    rows, decay = put(torch.cat([k.raw, k.beta], 1)), put(k.decay)
    got = [ops.delta_rule(rows[a:b, :C], ops.ShortConv(put(k.w), None, ring), rows[a:b, C:], decay[a:b], k.bias.to(device), k.A.to(device), S, 1,
                          128 ** -0.5, step_of([(a, b - a, 1)], None, device)).float().cpu() for a, b in ((0, T - 70), (T - 70, T))]
    close(torch.cat(got), k.want, dtype, LOOSE[dtype] * max(1.0, float(k.want.abs().max())))
    fault_free(device)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_recurrences_of_a_mixed_batch(device, dtype):
    """Portions and single tokens of several sequences in one step, slots in any order, a padding row, and a slot that another
    sequence used before."""
    H, P, N, G, taps = 4, 24, 16, 2, 4
    cases = [space_case(H, P, N, G, taps, 50, 100 * i) for i in range(4)]
    shared = cases[0]                                                       # weights are one layer's
    for c in cases[1:]:
        c.__dict__.update(w=shared.w, b=shared.b, A=shared.A, D=shared.D, dt_bias=shared.dt_bias)
    put = lambda t: t.to(device, dtype).contiguous()  # noqa: E731
    ring, S, _ = state_record(taps, shared.raw.shape[1], (H, P, N), dtype, device, slots=4)
    conv = ops.ShortConv(put(shared.w), put(shared.b), ring)
    C = shared.raw.shape[1]
    at, slot = [0] * 4, [3, 0, 2, 1]
    got = [[] for _ in cases]
    alone = []
    for c in cases:                                                         # the same op, each sequence alone in one portion
        r2, S2, _ = state_record(taps, C, (H, P, N), dtype, device, 1)
        alone.append(ops.state_space(put(c.raw), ops.ShortConv(conv.w, conv.bias, r2), put(c.dt), shared.dt_bias.to(device), shared.A.to(device),
                                     shared.D.to(device), S2, G, step_of([(0, 50, 0)], None, device)).float().cpu())
    for news in ([17, 1, 5, 0], [1, 9, 1, 30], [20, 40, 0, 1], [12, 0, 44, 19]):
        order = sorted((i for i in range(4) if news[i]), key=lambda i: news[i] <= 1)
        step = step_of([(at[i], news[i], slot[i]) for i in order], None, device)
        rows = put(torch.cat([torch.cat([cases[i].raw, cases[i].dt], 1)[at[i]:at[i] + news[i]] for i in order]))
        y = ops.state_space(rows[:, :C], conv, rows[:, C:], shared.dt_bias.to(device), shared.A.to(device), shared.D.to(device), S, G, step).float().cpu()
        k = 0
        for i in order:
            got[i].append(y[k:k + news[i]])
            k, at[i] = k + news[i], at[i] + news[i]
    for i in range(4):
        assert at[i] == 50
        close(torch.cat(got[i]), alone[i], dtype, max(1.0, float(alone[i].abs().max())))
    fault_free(device)


def test_recurrence_cases_notice():
    """The cases' memories are long enough that a lost state shows at the end."""
    k = space_case(6, 16, 24, 2, 3, 61, 30)
    q = delta_case(4, 2, 16, 24, 4, 61, 20)
    g = torch.exp(-q.A.double() * oracle.softplus(torch.tensor(-4.0).double()))
    assert float((g ** 61).max()) > 0.3
    a = torch.exp(-k.A * oracle.softplus(k.dt_bias))
    assert float((a ** 61).max()) > 0.2


# ------------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("count,far", [(16, 40), (32, 110), (10, 23), (32, 1000), (4, 9), (2, 5), (64, 65), (1, 10), (32, 128), (32, 256)])
def test_distance_buckets(count, far):
    rel = rand(0, count, 3)
    got = distance_biases(rel, far)
    for n in range(0, 3 * far):
        if count > 1:
            assert torch.equal(got[:, min(n, got.shape[1] - 1)], rel[oracle.bucket(n, count, far)])


def sigmoid_case(T, H, G, d, seed, point):
    """Queries that point at single keys: query t scores 8 on the key ``point(t)`` and about 0 on others, and with the heads' offsets
    of -6 the others together weigh little."""
    k = rand(seed, T, G, d)
    k = k / k.norm(dim=-1, keepdim=True) * 4
    q = rand(seed + 1, T, H, d) * 0.05
    for t in range(T):
        j = point(t)
        if j is not None and 0 <= j <= t:
            q[t] += k[j].repeat_interleave(H // G, 0) * 0.75
    rel = rand(seed + 2, 16, H)
    return q.bfloat16().float(), k.bfloat16().float(), rel, rand(seed + 3, H) * 0.3 - 6, rand(seed + 4, T, H, d)


def plain_attention(q, k, rel, pb, gate, scale, far, window, keep, factor):
    T, H, d = q.shape
    G = k.shape[1]
    out = []
    for a in range(H):
        kv = k[:, a // (H // G)].double()
        o = oracle.attend(q[:, a].double(), kv, kv, scale, lambda n: rel[oracle.bucket(n, rel.shape[0], far), a].double() + pb[a].double(),
                          window or T + 1, keep)
        out.append(o * oracle.sigmoid(gate[:, a].double()) * factor)
    return torch.cat(out, 1)


HEADS = [(1, 1, 8), (6, 2, 24), (8, 1, 64), (4, 4, 128), (6, 3, 88), (2, 1, 136), (40, 2, 16), (4, 2, 200), (3, 1, 256)]
MASKS = [(0, 0), (33, 0), (64, 20), (1, 1), (17, 130), (100, 5)]


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("H,G,d", HEADS)
def test_sigmoid_attention(device, dtype, H, G, d):
    T, bt, far, factor, scale = (300 if device == "cuda" else 90), 16, 37, 1.3, d ** -0.5 * 4
    for n, (window, keep) in enumerate(MASKS if device == "cuda" or (H, G) == (6, 2) else MASKS[2:3]):
        # targets: the newest hidden, the oldest seen, the last kept, the first not kept, page and tile borders
        aims = [lambda t: t - window, lambda t: t - window + 1, lambda t: keep - 1, lambda t: keep, lambda t: t // 128 * 128, lambda t: t // 16 * 16 - 1,
                lambda t: t, lambda t: 0]
        q, k, rel, pb, gate = sigmoid_case(T, H, G, d, 10 * n, lambda t: aims[t % len(aims)](t))
        want = plain_attention(q, k, rel, pb, gate, scale, far, window, keep, factor)
        D = up8(d)
        blocks = torch.randperm(T // bt + 8, generator=torch.Generator().manual_seed(n)).tolist()
        cache = torch.full((len(blocks), G, bt, D), NAN).to(device, dtype)
        bias = (distance_biases(rel, far) + pb[:, None]).to(device).contiguous()
        rows = torch.cat([pad(q, D).flatten(1), pad(k, D).flatten(1), pad(gate, D).flatten(1)], 1).to(device, dtype)
        nq, nk = H * D, G * D
        out, at = [], 0
        for size in [129, 1, 2, 40, 1, 100, 1, 1, 25] if T == 300 else [33, 1, 2, 40, 1, 12, 1]:
            step = make_step([(at, size)], [blocks[:T // bt + 1]], bt, device)
            part = rows[at:at + size]
            ops.panel_append(part[:, nq:nq + nk], step, cache, bt)
            wide = torch.zeros(size, nq + 8, device=device, dtype=dtype)
            w = ops.SigmoidWeights(bias, part[:, nq + nk:], factor)
            ops.panel_attention(part, cache, cache, bt, step, H, G, scale, window, keep, weights=w, out=wide[:, :nq])
            assert not wide[:, nq:].any()
            out.append(wide[:, :nq].unflatten(1, (H, D))[..., :d].flatten(1).float().cpu())
            at += size
        assert at == T
        close(torch.cat(out), want, dtype, max(1.0, float(want.abs().max())))
    fault_free(device)


@pytest.mark.parametrize("device,dtype", PLACES)
def test_sigmoid_attention_far_back(device, dtype):
    """One far key among hundreds, without a window: whole prompts over several tiles, and decoding that is split over CTAs. Batch of
    unequal sequences in one step, a padding sequence among the single tokens, no gate."""
    H, G, d, bt, far, scale = 4, 2, 64, 16, 50, 0.5
    lens = [700, 450, 513] if device == "cuda" else [120, 70, 65]
    cases = []
    for i, T in enumerate(lens):
        q, k, rel, pb, _ = sigmoid_case(T, H, G, d, 50 + 7 * i, lambda t: (t * 37) % max(t, 1))
        if i:
            rel, pb = cases[0][2:4]
        cases.append((q, k, rel, pb))
    rel, pb = cases[0][2:]
    bias = (distance_biases(rel, far) + pb[:, None]).to(device).contiguous()
    wants = [plain_attention(q, k, rel, pb, torch.full_like(q, 1e4), scale, far, 0, 0, 1.0) for q, k, _, _ in cases]
    tables, base = [], 0
    for T in lens:
        tables.append(list(range(base, base + T // bt + 1)))
        base += T // bt + 1
    cache = torch.full((base, G, bt, d), NAN).to(device, dtype)
    rows = [torch.cat([q.flatten(1), k.flatten(1)], 1).to(device, dtype) for q, k, _, _ in cases]
    got = [[] for _ in lens]
    at = [0] * len(lens)
    for rest in (2, 1, 0):
        news = [T - rest - a for T, a in zip(lens, at)]
        step = make_step(list(zip(at, news)), tables, bt, device)
        part = torch.cat([r[a:a + n] for r, a, n in zip(rows, at, news)])
        ops.panel_append(part[:, H * d:], step, cache, bt)
        o = ops.panel_attention(part, cache, cache, bt, step, H, G, scale, weights=ops.SigmoidWeights(bias)).float().cpu()
        c = 0
        for i, n in enumerate(news):
            got[i].append(o[c:c + n])
            c, at[i] = c + n, at[i] + n
    for g, w in zip(got, wants):
        close(torch.cat(g), w, dtype, max(1.0, float(w.abs().max())))
    fault_free(device)


def test_attention_cases_notice():
    q, k, rel, pb, gate = sigmoid_case(90, 6, 2, 24, 0, lambda t: [t - 20, t - 19, 4, 5][t % 4])
    args = (q, k, rel, pb, gate, 24 ** -0.5 * 4, 37)
    want = plain_attention(*args, 20, 5, 1.3)
    for window, keep in ((21, 5), (19, 5), (20, 4), (20, 6)):
        assert float((plain_attention(*args, window, keep, 1.3) - want).abs().max()) > 10 * TOL[torch.bfloat16] * max(1.0, float(want.abs().max()))


# ------------------------------------------------------------------------------------------------ experts
def apart(E, T, seed, top, count, keep):
    """Router logits whose choices do not hinge on rounding."""
    g = torch.Generator().manual_seed(seed)
    rows = []
    while len(rows) < T:
        z = torch.randn(E, generator=g) * 3
        groups = z.view(count, -1).max(-1).values.sort().values
        if keep < count and float(groups[-keep] - groups[-keep - 1]) < 1e-3:
            continue
        best = z.view(count, -1).max(-1).values.topk(keep).indices
        left = z.view(count, -1)[best].flatten().sort().values
        if top < len(left) and float(left[-top] - left[-top - 1]) < 1e-3:
            continue
        rows.append(z)
    return torch.stack(rows)


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("E,top,count,keep", [(15, 4, 5, 3), (10, 2, 1, 1), (9, 2, 3, 1), (5, 5, 1, 1), (64, 6, 8, 3), (40, 8, 40, 12), (1, 1, 1, 1), (2, 1, 2, 1),
                                              (512, 10, 64, 4)])
def test_choice_of_experts(device, E, top, count, keep):
    z = apart(E, 37, E + top, top, count, keep)
    logits = torch.cat([z, torch.full((37, 7), 50.0)], 1).to(device)                 # columns behind the experts' do not count
    ids, w = ops.moe_route(logits, top, scoring="softmax", renorm=True, n_group=count, topk_group=keep, E=E, group_top=1)
    for t in range(37):
        want = oracle.choose(z[t].double(), top, count, keep)
        got = {int(e): float(v) for e, v in zip(ids[t].cpu(), w[t].cpu())}
        assert got.keys() == want.keys()
        for e, v in want.items():
            assert abs(got[e] - float(v)) < 1e-5


def test_group_score_matters():
    """The best group by its largest score is not the best by the sum of its two largest."""
    z = torch.tensor([[3.0, -2.0, 2.5, 2.4, 0.0, 0.1]])
    for top, want in ((1, 0), (2, 2)):
        ids, _ = ops.moe_route(z, 1, scoring="softmax", renorm=True, n_group=3, topk_group=1, group_top=top)
        assert int(ids[0, 0]) == want


@pytest.mark.parametrize("device,dtype", PLACES)
@pytest.mark.parametrize("T,E,top,H,ff", [(1, 4, 2, 64, 24), (37, 14, 3, 72, 24), (300, 6, 2, 128, 40)])
def test_clamped_experts_beside_a_mixer(device, dtype, T, E, top, H, ff):
    """Expert outputs through the clamped unit, and their weighted sum plus the mixer's result (weight one) on the stream."""
    limit = 1.1
    x, wg, wu, wd = rand(0, T, H), rand(1, E, ff, H) * 0.3, rand(2, E, ff, H) * 0.3, rand(3, E, H, ff) * 0.2
    F = up8(ff)
    w13 = torch.cat([pad(wg.transpose(1, 2), F).transpose(1, 2), pad(wu.transpose(1, 2), F).transpose(1, 2)], 1).reshape(-1, H).to(device, dtype)
    w2 = pad(wd, F).reshape(-1, F).to(device, dtype)
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:top] for t in range(T)])
    wt = torch.rand(T, top, generator=torch.Generator().manual_seed(9))
    y, rows = expert_outputs(x.to(device, dtype), ids.to(torch.int32).to(device), w13, w2, F, MlpSpec(ff, limit))
    mixer, stream = rand(5, T, H), rand(6, T, H) * 3
    norm = ops.NormParams(torch.full((H,), 0.8).to(device, dtype), None, H, 1e-4, rms=True)
    out, z = ops.stream_add(stream.clone().to(device), ops.ExpertSum(y, rows, wt.to(device), mixer.to(device, dtype)), None, None, norm)
    want = stream.double() + mixer.double()
    for t in range(T):
        for j, e in enumerate(ids[t].tolist()):
            w = {"gate": wg[e].double(), "up": wu[e].double(), "down": wd[e].double()}
            want[t] += float(wt[t, j]) * oracle.expert(x[t].double(), w, "", limit)
    close(out, want, dtype)
    close(z, oracle.rms(want, 1e-4) * 0.8, dtype, 4.0)
    fault_free(device)
