"""The shared paged runtime (slots, pages, mixed-batch step) and the step scheduler, on the CPU with a stand-in model whose
logits reveal exactly which cached tokens a row can see through its page table."""
import random

import pytest
import torch

from deepseek_v4_2080ti_b200.cli.trace_run import TraceSession, replay
from deepseek_v4_2080ti_b200.models.paged import PagedRuntime
from deepseek_v4_2080ti_b200.runtime.step_scheduler import StepScheduler

VOCAB = 97


def _expected(history, chunk):
    """Hash of the tokens a row may look at: all of its chunk, or everything."""
    lo = (len(history) - 1) // chunk * chunk if chunk else 0
    h = 7
    for i, t in enumerate(history[lo:]):
        h = (h * 31 + t * (i + 3)) % 10007
    return h % VOCAB


class HistoryModel(PagedRuntime):
    """Caches token ids; the logits of a row point at a hash of the tokens its page table shows."""
    tile_min_rows = 4

    def __init__(self, chunk=0, **kw):
        super().__init__("cpu", **kw)
        self.chunk = chunk
        self.cache = torch.full((self.num_blocks * self.block_size,), -1, dtype=torch.int64)
        self.batches = []

    def history_floor(self, length):
        return length - length % self.chunk if self.chunk else 0

    def history_span(self):
        return self.chunk - 1 if self.chunk else None

    def _next(self, logits):
        return logits.argmax(-1).to(torch.int32)

    def _forward(self, ids, positions, kv_slots, meta, rows):
        self.cache[kv_slots.long()] = ids.long()
        t = ids.numel()
        tables = meta["block_table"] if meta["mode"] == "decode" else self.block_table[meta["row_seq"].long()]
        if meta["mode"] == "mixed":
            assert meta["tile_rows"] == (sum(meta["q_len"].tolist()) if meta["tile_rows"] else 0)
        self.batches.append((meta["mode"], t))
        out = torch.zeros(t, VOCAB)
        for r in range(t):
            p = int(positions[r])
            hist = [int(self.cache[int(tables[r][j // self.block_size]) * self.block_size + j % self.block_size])
                    for j in range(self.history_floor(p), p + 1)]
            out[r, _expected([0] * self.history_floor(p) + hist, self.chunk)] = 1.0
        return out if rows is None else out[rows.long()] if rows.numel() else None


def _prompt(rng, n):
    return [rng.randrange(VOCAB) for _ in range(n)]


@pytest.mark.parametrize("chunk", [0, 5, 8, 21])
def test_mixed_steps_see_their_own_history_and_give_pages_back(chunk):
    rng = random.Random(chunk)
    rt = HistoryModel(chunk, max_slots=3, max_context=64, block_size=8, num_blocks=25)
    live, fed = {}, 0
    for step in range(300):
        while len(live) < 3 and rng.random() < 0.5:
            live[rt.allocate()] = []
        entries, want = [], []
        for slot, hist in live.items():
            if rng.random() < 0.3:
                continue                                     # left out of this step, goes on later
            n = min(rng.choice([1, 1, 2, 3, 5, 9, 17]), 64 - len(hist))
            if n <= 0:
                continue
            toks = _prompt(rng, n)
            places = sorted(rng.sample(range(n), rng.randint(0, n)))
            entries.append((slot, toks, places))
            want += [_expected(hist + toks[:w + 1], chunk) for w in places]
            hist += toks
            fed += n
        if entries:
            logits = rt.step(entries)
            got = [] if logits is None else logits.argmax(-1).tolist()
            assert got == want
        for slot in [s for s, h in live.items() if len(h) >= 64 or rng.random() < 0.05]:
            rt.free(slot)
            live.pop(slot)
        held = [b for st in rt.seqs.values() for b in st.blocks if b]
        assert len(held) == len(set(held)) and len(held) + len(rt.free_blocks) == rt.num_blocks - 1
        for st in rt.seqs.values():
            assert sum(b != 0 for b in st.blocks) <= rt.pages_held(max(st.length, 1), 17)
    for slot in list(live):
        rt.free(slot)
    assert fed > 500 and sorted(rt.free_blocks) == list(range(1, 25)) and all(r == 0 for r in rt.block_refs)


def test_a_step_that_does_not_fit_leaves_the_sequence_usable():
    rt = HistoryModel(0, max_slots=2, max_context=64, block_size=8, num_blocks=5)
    a, b = rt.allocate(), rt.allocate()
    with pytest.raises(RuntimeError, match="no free slot"):
        rt.allocate()
    rt.step([(a, list(range(20)), [])])
    with pytest.raises(RuntimeError, match="exhausted"):
        rt.step([(b, list(range(20)), [19])])
    rt.free(a)
    assert rt.step([(b, list(range(20)), [19])]).argmax(-1).tolist() == [_expected(list(range(20)), 0)]
    with pytest.raises(RuntimeError, match="max_context"):
        rt.step([(b, [1] * 60, [])])


def _greedy(prompt, n, chunk, eos=()):
    hist, out = list(prompt), []
    while len(out) < n:
        out.append(_expected(hist, chunk))
        if out[-1] in eos:
            return out[:-1], "stop"
        hist.append(out[-1])
    return out, "length"


@pytest.mark.parametrize("chunk,pool", [(0, 40), (0, 14), (6, 40), (6, 9)])
def test_scheduler_matches_each_request_alone(chunk, pool):
    rng = random.Random(pool + chunk)
    rt = HistoryModel(chunk, max_slots=3, max_context=96, block_size=8, num_blocks=pool)
    reqs = [(_prompt(rng, rng.randint(1, 60)), rng.randint(1, 25)) for _ in range(12)]
    sched = StepScheduler(rt, eos_ids={5}, max_batch=3, token_budget=16)
    for i, (p, n) in enumerate(reqs):
        sched.submit(i, p, n)
    res = sched.run()
    for i, (p, n) in enumerate(reqs):
        assert res[i][:2] == _greedy(p, n, chunk, {5}), i
        assert res[i][2]["total_seconds"] >= 0
    assert sched.mixed_rounds > 0 and max(t for _, t in rt.batches) <= 16
    assert len(rt.free_slots) == 3 and len(rt.free_blocks) == pool - 1


def test_scheduler_refuses_what_can_never_run():
    rt = HistoryModel(0, max_slots=2, max_context=64, block_size=8, num_blocks=5)
    sched = StepScheduler(rt)
    with pytest.raises(ValueError):
        sched.submit(0, [], 4)
    with pytest.raises(ValueError, match="context"):
        sched.submit(0, [1] * 60, 10)
    with pytest.raises(ValueError, match="pages"):
        sched.submit(0, [1] * 30, 10)


def test_adapter_batches_through_the_step_scheduler():
    from deepseek_v4_2080ti_b200.runtime.loader import GgufRuntimeAdapter
    rt = HistoryModel(0, max_slots=2, max_context=64, block_size=8)
    ad = GgufRuntimeAdapter(rt, 64, 2, "cpu")
    prompts = [[1, 2, 3, 4, 5, 6, 7], [9], [11, 12]]
    res = ad.generate_batch(prompts, [6, 9, 3], set(), 2)
    assert [r[0] for r in res] == [_greedy(p, n, 0)[0] for p, n in zip(prompts, [6, 9, 3])]
    s = ad.allocate()
    t = ad.prefill_tokens(s, prompts[0], 3, None)
    assert t == res[0][0][0] and ad.decode_tokens([s], [t], None) == [res[0][0][1]]
    ad.free(s)


def test_trace_replay_writes_wanted_logits_and_reuses_slots(tmp_path):
    import io
    import json

    import numpy as np
    rt = HistoryModel(0, max_slots=1, max_context=32, block_size=8)
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": [3, 4, 5], "want": [0, 2]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": [6], "want": []}], "end": ["a"]}),
             json.dumps({"step": 2, "entries": [{"id": "b", "tokens": [8, 9], "want": [1]}], "end": ["b"]})]
    done = io.StringIO()
    replay(rt, lines, str(tmp_path), done)
    assert done.getvalue().split("\n") == ["done 0", "done 1", "done 2", ""]
    assert sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "2.f32"]
    got = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, VOCAB).argmax(-1).tolist()
    assert got == [_expected([3], 0), _expected([3, 4, 5], 0)]
    assert np.fromfile(tmp_path / "2.f32", dtype="<f4").reshape(1, VOCAB).argmax(-1).tolist() == [_expected([8, 9], 0)]
    assert not TraceSession(rt).slots and rt.free_slots == [0]
