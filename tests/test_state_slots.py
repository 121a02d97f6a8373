"""State that sequences hold as a whole beside their blocks: the C++ scheduler's slots, without a model. A slot's content is
modelled as the list of tokens that went through it; before every step each running sequence's slot must hold exactly the
tokens that its cached length says, whatever forks, beams, preemptions and reuse happened in between."""
import numpy as np
import pytest

from ksanallm_b200.utils import native_engine as ne
from test_scheduler import cfg, make


class Slots:
    """Executes the state operations of step plans."""

    def __init__(self, device, host):
        self.device, self.host = [["stale", i] for i in range(device)], [None] * host

    def apply(self, plan):
        pairs = [np.asarray(getattr(plan, k)).reshape(-1, 2).tolist() for k in ("state_copies", "state_out", "state_in")]
        copies, out, back = pairs
        assert not {s for s, _ in copies} & {d for _, d in copies} and len({d for _, d in copies}) == len(copies)
        for s, d in copies:
            self.device[d] = list(self.device[s])
        for s, h in out:
            self.host[h] = list(self.device[s])
            self.device[s] = ["swapped"]
        for s, h in back:
            self.device[s] = list(self.host[h])
            self.host[h] = None

    def run(self, s, plan):
        """Feeds the plan's rows through their slots; no two sequences may share one."""
        slots = plan.state_slots.tolist()
        assert len(set(slots)) == len(slots) == len(plan.seq_ids) and min(slots, default=0) >= 0
        at = 0
        for sid, n, kv, slot in zip(plan.seq_ids.tolist(), plan.q_lens.tolist(), plan.kv_lens.tolist(), slots):
            if kv - n > 0:
                assert self.device[slot] == s.get_tokens(sid)[:kv - n], (sid, slot)
            else:
                self.device[slot] = []
            self.device[slot] = self.device[slot] + plan.input_ids[at:at + n].tolist()
            at += n


def drive(s, slots, rng, beams=(), steps=4000, hook=None):
    done, n = {}, 0
    while not s.idle() and n < steps:
        n += 1
        plan = s.schedule()
        for ev in plan.events:
            done[ev[0]] = ev[5]
        slots.apply(plan)
        if plan.empty():
            continue
        again = ne.StepPlan.unpack(plan.pack())
        for k in ("state_slots", "state_copies", "state_out", "state_in", "block_table", "seq_ids"):
            assert np.array_equal(getattr(again, k), getattr(plan, k)), k
        slots.run(s, plan)
        ids = plan.sample_seq_ids.tolist()
        tokens = [int(rng.integers(10, 9999)) for _ in ids]
        parents = []
        for sid in ids:
            group = next((g for g in beams if sid in g), ())
            there = [x for x in group if x in ids and x in running(plan)]
            parents.append(int(rng.choice(there)) if len(there) == len(group) > 0 else -1)
        for ev in s.post_step(plan, tokens, parents):
            if ev[4]:
                done[ev[0]] = ev[5]
        if hook:
            hook(n)
        ok, why = s.check_invariants()
        assert ok, why
    assert s.idle()
    return done


def running(plan):
    return set(plan.seq_ids.tolist())


@pytest.mark.parametrize("seed", range(4))
@pytest.mark.parametrize("mode,host", [(0, 60), (0, 6), (1, 0)], ids=["swap", "swap-small", "recompute"])
def test_slots_follow_their_sequences(mode, host, seed):
    rng = np.random.default_rng(seed)
    slots = Slots(6, 6 if host else 0)
    s = make(24, host, max_batch_size=6, num_state_slots=6, num_host_state_slots=6 if host else 0, preempt_mode=mode,
             split_fuse_token_num=int(rng.integers(0, 2)) * 18, enable_prefix_cache=True)
    want = {}
    for r in range(14):
        _, _, ids = s.add_request(r, rng.integers(10, 9999, int(rng.integers(1, 50))).tolist(),
                                  cfg(int(rng.integers(1, 40)), num_return_sequences=int(rng.integers(1, 4))))
        want.update(dict.fromkeys(ids))
    drop = rng.integers(0, 14)
    done = drive(s, slots, rng, hook=lambda n: s.abort(int(drop)) if n == 9 else None)
    assert set(done) == set(want)
    st = s.stats()
    assert (st["preempt_swap"] if mode == 0 else st["preempt_recompute"]) > 0 and st["prefix_hit_tokens"] == 0
    assert st["used_blocks"] == 0


@pytest.mark.parametrize("seed", range(6))
def test_beams_exchange_states(seed):
    """Random parents: permutations, one parent for all, chains. Eight slots for groups of three and four beams and a single."""
    rng = np.random.default_rng(100 + seed)
    s = make(200, 0, max_batch_size=8, num_state_slots=8, preempt_mode=1)
    beams = []
    for r, n in enumerate((3, 4, 1, 4, 3)):
        _, _, ids = s.add_request(r, rng.integers(10, 9999, int(rng.integers(1, 30))).tolist(), cfg(25, num_beams=n, logprobs_num=n))
        if n > 1:
            beams.append(tuple(ids))
    done = drive(s, Slots(8, 0), rng, beams)
    assert len(done) == 15 and all(code == 0 for code in done.values())


def test_replaced_tokens_start_over():
    """A state cannot be rolled back: a sequence whose generated tokens are replaced is computed again from its start."""
    rng = np.random.default_rng(1)
    s = make(50, 0, max_batch_size=2, num_state_slots=2, preempt_mode=1)
    _, _, (sid,) = s.add_request(0, list(range(100, 120)), cfg(12))
    slots = Slots(2, 0)

    def replace(n):
        if n == 5:
            kept = s.get_tokens(sid)[20:]
            s.replace_generated(sid, kept[:2] + [7, 8])

    drive(s, slots, rng, hook=replace)


def test_requests_without_a_slot_wait():
    s = make(50, 0, max_batch_size=8, num_state_slots=2, preempt_mode=1)
    rng = np.random.default_rng(2)
    for r in range(5):
        s.add_request(r, list(range(10, 20 + r)), cfg(3 + r))
    plan = s.schedule()
    assert len(plan.seq_ids) == 2
    slots = Slots(2, 0)
    slots.apply(plan)
    slots.run(s, plan)
    s.post_step(plan, [11, 12])
    assert len(drive(s, slots, rng)) == 5


def test_plans_without_state_carry_none():
    s = make(50, 0)
    s.add_request(0, [1, 2, 3], cfg(2))
    plan = s.schedule()
    assert plan.state_slots.size == plan.state_copies.size == plan.state_out.size == plan.state_in.size == 0
