"""The Kemirax runtime on the GPU against the plain whole-sequence statement: prompts, token-by-token decoding, portions, mixed
batches, reused pages and state slots, far keys and long memories, and the public entry points; and the boundary step, the
routing and the expert kernels it uses."""
import random

import pytest
import torch

from deepseek_v4_2080ti_b200.models import kemirax as kx
from deepseek_v4_2080ti_b200.models.reference_cpu import kemirax_ref as ref

pytestmark = pytest.mark.gpu
F32_TOL = 4e-5
M, G, E, L = kx.LatentSpec, kx.LinearSpec, kx.ExpertsSpec, kx.LayerSpec
YARN = {"factor": 3.0, "original": 64, "fast": 4.0, "slow": 0.5}

CONFIGS = {
    # nothing is a multiple of anything; both mixers with and without a feed-forward, a borrower far behind its lender
    "ragged": kx.KemiraxConfig(211, 84, 1e-3, [
        L(G(3, 20, 28, 6.0, 7), E(22, 1.2, 5, 2, 3, 41, 0.7)), L(M(5, 20, 6, 12, 33, 40, 0.3, 6, 500.0, YARN)), L(G(1, 52, 9, 1.0, 30)),
        L(M(3, 12, 6, 30, 17, 40, 0.25, 6, 500.0, YARN, kv_from=1), E(19, 0.6, 3, 1, 2, 8, 1.5))]),
    # plain rotation over part of the key, no shared expert, no identity expert, one expert per token; two borrowers
    "borrow": kx.KemiraxConfig(128, 128, 1e-6, [
        L(M(4, 64, 32, 64, 48, 64, 0.1, 16, 10000.0), E(64, 4.0, 8, 0, 1)), L(M(2, 16, 32, 96, 64, 64, 0.2, 16, 10000.0, kv_from=0), E(64, 1.0, 4, 4, 5, 64, 1.0)),
        L(M(6, 32, 32, 32, 16, 64, 0.15, 16, 10000.0, kv_from=0), E(32, 2.0, 1, 1, 1, 16, 2.0))]),
    # heads wider than the tile kernel takes: every row goes through the absorbed form
    "wide": kx.KemiraxConfig(97, 64, 1e-5, [
        L(M(2, 200, 80, 144, 40, 176, 0.06, 80, 2000.0, YARN), E(48, 2.0, 3, 1, 2, 24, 1.0)), L(G(2, 130, 40, 16.0, 16), E(16, 1.0, 2, 0, 2))]),
    # recurrent only: no pages are ever read
    "recurrent": kx.KemiraxConfig(160, 96, 1e-5, [L(G(2, 64, 64, 16.0, 16), E(40, 1.5, 6, 2, 4, 48, 1.0)), L(G(4, 16, 32, 8.0, 8)), L(G(1, 32, 16, 2.0, 16))]),
}


class Case:
    """A runtime and the statement's logits for whole sequences (cached per sequence)."""

    def __init__(self, name, dtype, slots=4, context=512, blocks=None, block_size=64, change=None):
        self.cfg, self.dtype = CONFIGS[name], dtype
        self.state = dict(kx.synth_state(self.cfg, seed=len(name)))
        if change:
            change(self.state)
        self.rt = kx.KemiraxRuntime(self.cfg, kx.KemiraxWeights(self.cfg, self.state, "cuda", dtype), max_slots=slots,
                                    max_context=context, num_blocks=blocks, block_size=block_size)
        for i in range(len(self.cfg.layers)):        # what earlier requests may have left: nothing of it may show
            if self.rt.cache[i] is not None:
                self.rt.cache[i][1:] = 60.0
            if self.rt.state[i] is not None:
                self.rt.state[i].fill_(float("nan"))
            self.rt.tails[i].fill_(float("nan"))
        self.raw, self.memo = self.cfg.to_json(), {}

    def want(self, toks):
        key = tuple(toks)
        if key not in self.memo:
            self.memo[key] = ref.forward(self.raw, self.state, toks, torch.float64)
        return self.memo[key]

    def near(self, got, want, tol=None):
        """Row errors relative to the spread of the logits.  In bf16 a token may choose another expert where two scores are
        equal within rounding: a few rows may be off by more."""
        d = got.double().cpu() - want
        d = d - d.mean(-1, keepdim=True)
        err = d.pow(2).mean(-1).sqrt() / want.std()
        if tol or self.dtype == torch.float32:
            assert float(err.max()) < (tol or F32_TOL), (float(err.max()), int(err.argmax()))
        else:
            over = int((err > 6e-2).sum())
            assert over <= max(1, err.numel() // 20) and float(err.median()) < 3e-2, (over, float(err.max()), float(err.median()))

    def feed(self, slot, toks, cuts):
        """All logits of a sequence fed in the given portions."""
        rows, at = [], 0
        for n in cuts:
            rows.append(self.rt.step([(slot, toks[at:at + n], list(range(n)))]).clone())
            at += n
        assert at == len(toks)
        return torch.cat(rows)


def _tokens(cfg, n, seed=0):
    rng = random.Random(seed)
    return [rng.randrange(cfg.vocab) for _ in range(n)]


BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
ALL = pytest.mark.parametrize("name", sorted(CONFIGS))


@BOTH
@ALL
def test_layers_and_logits_of_a_whole_prompt(name, dtype):
    from deepseek_v4_2080ti_b200.ops import _lib
    c = Case(name, dtype)
    toks = _tokens(c.cfg, 203, seed=1)
    taps, want_taps = [], []
    c.rt.residual_tap = lambda i, x: taps.append((i, x.cpu()))
    slot = c.rt.allocate()
    got = c.rt.step([(slot, toks, list(range(203)))])
    _lib.check_status()
    want = ref.forward(c.raw, c.state, toks, torch.float64, want_taps)
    assert [i for i, _ in taps] == list(range(len(c.cfg.layers)))
    for (_, x), y in zip(taps, want_taps):
        err = (x.double() - y).norm(dim=-1) / y.norm(dim=-1)
        assert float(err.max() if dtype == torch.float32 else err.median()) < (1e-5 if dtype == torch.float32 else 2e-2)
    c.near(got, want)
    assert (c.rt.tile_min_rows < 100) == (dtype == torch.bfloat16 and name != "wide")
    c.rt.free(slot)
    c.rt.residual_tap = None
    slot = c.rt.allocate()                            # with and without the tap: the same numbers
    c.near(c.rt.step([(slot, toks, list(range(203)))]), got.double().cpu(), 1e-6 if dtype == torch.float32 else 1e-2)
    c.rt.free(slot)


@BOTH
@ALL
def test_token_by_token_equals_the_prompt(name, dtype):
    c = Case(name, dtype)
    toks = _tokens(c.cfg, 140, seed=2)
    slot = c.rt.allocate()
    c.near(c.feed(slot, toks, [1] * 140), c.want(toks))
    c.rt.free(slot)
    slot = c.rt.allocate()                            # the same slot and pages again
    c.near(c.feed(slot, toks, [27] + [1] * 113), c.want(toks))
    c.rt.free(slot)


@BOTH
@ALL
@pytest.mark.parametrize("size", [2, 3, 17, 50, 64])
def test_portions(name, dtype, size):
    c = Case(name, dtype)
    toks = _tokens(c.cfg, 155, seed=3)
    slot = c.rt.allocate()
    cuts = [size] * (155 // size) + ([155 % size] if 155 % size else [])
    c.near(c.feed(slot, toks, cuts), c.want(toks))


@pytest.mark.parametrize("block_size", [16, 32, 128])
def test_other_page_sizes(block_size):
    c = Case("ragged", torch.bfloat16, block_size=block_size)
    toks = _tokens(c.cfg, 190, seed=4)
    slot = c.rt.allocate()
    c.near(c.feed(slot, toks, [100, 2, 30, 1, 1, 56]), c.want(toks))


@BOTH
@ALL
def test_mixed_batches_with_reused_pages_and_slots(name, dtype):
    """Unequal requests beside each other in a pool too small for all of them, slots and pages used again and again."""
    from deepseek_v4_2080ti_b200.ops import _lib
    c = Case(name, dtype, slots=3, context=256, blocks=12)
    rng = random.Random(9)
    seqs = [_tokens(c.cfg, n, seed=20 + n) for n in (200, 5, 1, 130, 64, 65, 33, 90, 2)]
    todo, live, rows = list(range(len(seqs))), {}, {i: [] for i in range(len(seqs))}
    while todo or live:
        while todo and len(live) < 3 and c.rt.free_slots:
            held = sum((len(seqs[i]) + 63) // 64 for i in live)
            if held + (len(seqs[todo[0]]) + 63) // 64 > 11:
                break
            live[todo.pop(0)] = [c.rt.allocate(), 0]
        entries, owners = [], []
        for i, (slot, at) in live.items():
            if rng.random() < 0.15:
                continue
            n = min(rng.choice([1, 1, 1, 2, 9, 31, 70]), len(seqs[i]) - at)
            entries.append((slot, seqs[i][at:at + n], list(range(n))))
            owners += [i] * n
            live[i][1] += n
        if not entries:
            continue
        logits = c.rt.step(entries)
        for r, i in enumerate(owners):
            rows[i].append(logits[r].clone())
        for i in [i for i, (_, at) in live.items() if at == len(seqs[i])]:
            c.rt.free(live.pop(i)[0])
    _lib.check_status()
    for i, s in enumerate(seqs):
        c.near(torch.stack(rows[i]), c.want(s))
    assert len(c.rt.free_blocks) == 11 and len(c.rt.free_slots) == 3


@BOTH
@ALL
def test_first_tokens_and_single_token_requests(name, dtype):
    c = Case(name, dtype)
    for n in (1, 2, 3):
        toks = _tokens(c.cfg, n, seed=30 + n)
        for cuts in ([n], [1] * n):
            slot = c.rt.allocate()
            c.near(c.feed(slot, toks, cuts), c.want(toks))
            c.rt.free(slot)


@BOTH
def test_long_decoding(dtype):
    c = Case("ragged", dtype, slots=1, context=512)
    toks = _tokens(c.cfg, 420, seed=5)
    slot = c.rt.allocate()
    c.near(c.feed(slot, toks, [40] + [1] * 380), c.want(toks))


@BOTH
def test_a_far_token_shows(dtype):
    """Sharp attention and slow decays: another token far back gives other logits hundreds of positions later, and the runtime
    follows, in one portion, in several and decoding."""
    def change(state):
        state["l0.mix.a2.b"] += 8.0
        state["l2.mix.a2.b"] += 10.0
        for n in ("l1.mix.uk", "l1.mix.dkv", "l3.mix.uk"):
            state[n] *= 3.0
    c = Case("ragged", dtype, change=change)
    loud = c.state["embed"].float().norm(dim=-1).argmax().item()
    toks = [x if x != loud else (loud + 1) % c.cfg.vocab for x in _tokens(c.cfg, 330, seed=8)]
    with_it = [toks[0], loud] + toks[2:]
    w0, w1 = c.want(toks), c.want(with_it)
    assert float((w0[300:] - w1[300:]).pow(2).mean().sqrt() / w1.std()) > 0.02          # the far token shows
    for cuts in ([330], [70, 2, 1, 1, 200, 56], [290] + [1] * 40):
        slot = c.rt.allocate()
        c.near(c.feed(slot, with_it, cuts), w1)
        c.rt.free(slot)


@ALL
def test_greedy_decode_graph_and_eager_and_statement(name):
    c = Case(name, torch.float32)
    prompt = _tokens(c.cfg, 31, seed=6)
    hist = list(prompt)
    for _ in range(24):
        hist.append(int(c.want(hist)[-1].argmax()))
    ids = torch.tensor(prompt, dtype=torch.int32)
    assert c.rt.generate(ids, 24, chunk=9) == hist[31:]
    assert c.rt.generate(ids, 24, use_graph=False) == hist[31:]


@BOTH
def test_capturing_a_decode_graph_does_not_advance_the_state(dtype):
    """Two requests decode, a third joins: the batch sizes' graphs are captured in the middle of running sequences."""
    c = Case("recurrent", dtype)
    toks = [_tokens(c.cfg, 30, seed=70 + i) for i in range(3)]
    slots = [c.rt.allocate() for _ in range(3)]
    got = {i: [c.rt.step([(slots[i], toks[i][:20], [19])])[0].clone()] for i in range(3)}
    for p in range(20, 30):
        group = [0, 1] if p < 24 else [0, 1, 2]
        for i, row in zip(group, c.rt.step([(slots[i], [toks[i][p if i < 2 else p - 4]], [0]) for i in group])):
            got[i].append(row.clone())
    for i in range(3):
        c.near(torch.stack(got[i]), c.want(toks[i])[19:19 + len(got[i])])


def test_scheduler_batches_match_each_request_alone():
    from deepseek_v4_2080ti_b200.runtime.step_scheduler import StepScheduler
    c = Case("ragged", torch.float32, slots=3, context=256, blocks=10)
    reqs = [(_tokens(c.cfg, n, seed=40 + n), m) for n, m in ((70, 12), (3, 40), (1, 25), (120, 9), (20, 20), (64, 64))]
    sched = StepScheduler(c.rt, (), max_batch=3, token_budget=48)
    for i, (p, m) in enumerate(reqs):
        sched.submit(i, p, m)
    res = sched.run()
    assert sched.mixed_rounds > 0
    for i, (p, m) in enumerate(reqs):
        assert res[i][0] == c.rt.generate(torch.tensor(p, dtype=torch.int32), m), i


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_public_api_serves_a_checkpoint_folder(tmp_path, dtype):
    from pocketllm import LLM, EngineArgs, SamplingParams
    cfg = CONFIGS["ragged"]
    kx.write_checkpoint(str(tmp_path), cfg, seed=4)
    prompts = [_tokens(cfg, n, seed=50 + n) for n in (45, 4, 18)]
    llm = LLM(EngineArgs(model=str(tmp_path), max_model_len=256, max_batch_size=3, dtype=dtype))
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=10))
    one = llm.generate([{"prompt_token_ids": prompts[0]}], SamplingParams(max_tokens=10))[0]
    if dtype == "float32":
        state = dict(kx.synth_state(cfg, 4))
        for p, o in zip(prompts, outs):
            hist = list(p)
            for _ in range(10):
                hist.append(int(ref.forward(cfg.to_json(), state, hist, torch.float64)[-1].argmax()))
            assert list(o.token_ids) == hist[len(p):]
        assert list(one.token_ids) == list(outs[0].token_ids)
    assert all(len(o.token_ids) == 10 and max(o.token_ids) < cfg.vocab for o in outs)
    drawn = llm.generate([{"prompt_token_ids": prompts[1]}], SamplingParams(max_tokens=6, temperature=0.8, top_k=20, seed=7))[0]
    again = llm.generate([{"prompt_token_ids": prompts[1]}], SamplingParams(max_tokens=6, temperature=0.8, top_k=20, seed=7))[0]
    assert list(drawn.token_ids) == list(again.token_ids)
    lp = llm.generate([{"prompt_token_ids": prompts[1]}], SamplingParams(max_tokens=2, logprobs=True, top_logprobs=3))[0]
    assert len(lp.logprobs) == 2 and len(lp.logprobs[0]["top_logprobs"]) == 3
    llm.close()
    llm = LLM(EngineArgs(model="synthetic:kemirax-tiny", max_model_len=128, max_batch_size=2))
    assert len(llm.generate([{"prompt_token_ids": [1, 2, 3]}], SamplingParams(max_tokens=5))[0].token_ids) == 5
    llm.close()


def test_command_lines(tmp_path, capsys, monkeypatch):
    import io
    import json

    import numpy as np

    from deepseek_v4_2080ti_b200.cli import generate_gguf, trace_run
    cfg = CONFIGS["ragged"]
    kx.write_checkpoint(str(tmp_path / "m"), cfg, seed=2)
    state, raw = dict(kx.synth_state(cfg, 2)), cfg.to_json()
    toks = _tokens(cfg, 150, seed=61)
    want = ref.forward(raw, state, toks, torch.float64)
    assert generate_gguf.main(["--checkpoint", str(tmp_path / "m"), "--dtype", "float32", "--max-new-tokens", "1",
                               "--max-context", "256", "--token-ids", ",".join(map(str, toks))]) == 0
    out = capsys.readouterr().out
    assert f"tokens={int(want[-1].argmax())}\n" in out and "family=kemirax" in out
    (tmp_path / "o").mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:100], "want": [99, 0]}, {"id": "y", "tokens": toks[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[1:2], "want": [0]}, {"id": "x", "tokens": toks[100:], "want": [49]}], "end": ["y", "x"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert trace_run.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "256"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1"]
    for n, places in ((0, [99, 0]), (1, [1, 149])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", dtype="<f4").copy()).view(2, cfg.vocab).double()
        assert float((got - want[places]).abs().max() / want.std()) < 2e-4


# ---------------------------------------------------------------------------------------------- boundary step, routing, experts
DT = {torch.bfloat16: 1.2e-2, torch.float32: 3e-6}


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-30))


def _segments(entries):
    from deepseek_v4_2080ti_b200.ops.scan import Segments
    i32 = lambda v: torch.tensor(v, dtype=torch.int32).cuda()
    first, at = [], 0
    for _, n in entries:
        first.append(at)
        at += n
    rows = [(f, s) for f, (s, n) in zip(first, entries) for _ in range(n)]
    lens = [n for _, n in entries]
    return Segments(i32([f for f, _ in rows]), i32([s for _, s in rows]), i32(first), i32(lens), i32([s for s, _ in entries]), max(lens), min(lens))


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("cols,single", [(20, True), (333, False), (4112, True), (4112, False), (9000, False)])
def test_boundary_step(dtype, cols, single):
    """Everything the residual takes between two layers at once, the norm with one weight, and the shift across portions."""
    from deepseek_v4_2080ti_b200.ops import decoder as dec
    entries = [(2, 1), (0, 1), (4, 1)] if single else [(2, 5), (0, 1), (4, 2), (1, 9)]
    pos0 = {2: 7, 0: 0, 4: 3, 1: 0}
    n, ld, eps, top, real = sum(k for _, k in entries), dec.pad16(cols), 1e-3, 5, 6
    gen = torch.Generator().manual_seed(cols)
    r = lambda *s: torch.randn(*s, generator=gen)
    pad = lambda t, dt: torch.nn.functional.pad(t, (0, ld - t.shape[-1])).to("cuda", dt).contiguous()
    x, mix, h, shared = r(n, cols), r(n, cols).to(dtype), r(n, cols).to(dtype), r(n, cols).to(dtype)
    gates, gb, shift = r(n, 2, cols).to(dtype), r(2, cols), torch.rand(cols, generator=gen)
    idx = torch.stack([torch.randperm(real + 3, generator=gen)[:top] for _ in range(n)]).to(torch.int32)      # three identity experts
    wts = torch.rand(n, top, generator=gen)
    row = torch.full((n, top), -1, dtype=torch.int32)
    order = torch.randperm(n * top, generator=gen).to(torch.int32).view(n, top)
    row[idx < real] = order[idx < real]
    y = r(n * top, cols).to(dtype)
    sg = r(n, 3)
    tail = r(5, cols).to(dtype)
    want_x = x.double() + mix.double() * ref.sigmoid(gates[:, 0].double() + gb[0].double())
    ff = ref.sigmoid(sg[:, 1:2].double()) * shared.double()
    for t in range(n):
        for k in range(top):
            ff[t] += wts[t, k].double() * (y[row[t, k]] if idx[t, k] < real else h[t]).double()
    want_x = want_x + ff * ref.sigmoid(gates[:, 1].double() + gb[1].double())
    want_h = ref.rms(want_x, eps) * 1.7
    xg, tg = pad(x, torch.float32), pad(tail, dtype)
    pos = torch.tensor([pos0[s] + j for s, k in entries for j in range(k)], dtype=torch.int32).cuda()
    gpad = torch.nn.functional.pad(gates, (0, ld - cols)).reshape(n, 2 * ld)
    gpad = torch.nn.functional.pad(gpad, (0, 16)).to("cuda")
    seg = _segments(entries)
    kw = dict(ld=ld, n=n, dtype=dtype, mix=pad(mix, dtype), gates=gpad, gate_b=pad(gb, torch.float32).view(-1), h=pad(h, dtype),
              routed=dec.Routed(torch.nn.functional.pad(pad(y, dtype), (0, 16)), row.cuda(), idx.cuda(), wts.cuda(), real),
              shared=pad(shared, dtype), shared_gate=sg.cuda()[:, 1:])
    want_rows = torch.tensor([n - 1, 0], dtype=torch.int32).cuda()
    some, none = dec.parallel_step(xg, cols, 1.7, eps, **kw, rows=want_rows)
    assert none is None and _rel(some[:, :cols], want_h[[n - 1, 0]]) < DT[dtype] and torch.equal(xg, pad(x, torch.float32))
    hg, mg = dec.parallel_step(xg, cols, 1.7, eps, **kw, x_out=xg, shift=pad(shift, torch.float32), tail=tg, seg=seg, positions=pos)
    assert _rel(xg[:, :cols], want_x) < (2e-6 if dtype == torch.float32 else 1e-5) and not xg[:, cols:].any()
    assert _rel(hg[:, :cols], want_h) < DT[dtype] and not hg[:, cols:].any() and not mg[:, cols:].any()
    hq, at = hg[:, :cols].double().cpu(), 0                           # the shift works on the rounded norm
    for s, k in entries:
        before = tail[s].double() if pos0[s] else torch.zeros(cols).double()
        for t in range(at, at + k):
            assert _rel(mg[t, :cols], hq[t] + (before - hq[t]) * shift.double()) < DT[dtype], (s, t)
            before = hq[t]
        assert torch.equal(tg[s, :cols].double().cpu(), hq[at + k - 1])
        at += k
    assert torch.equal(tg[3, :cols].cpu(), tail[3])                    # nobody's slot
    # a layer without a feed-forward, and an embedding row as the start
    table, ids = r(9, cols).to(dtype), torch.tensor([8, 0, 3], dtype=torch.int32)
    x2 = torch.full((3, ld), 5.0).cuda()
    h2, _ = dec.parallel_step(None, cols, 0.5, eps, ld=ld, n=3, dtype=dtype, ids=ids.cuda(), table=pad(table, dtype), x_out=x2)
    assert _rel(x2[:, :cols], table[ids.long()].double()) < 1e-7 and _rel(h2[:, :cols], ref.rms(table[ids.long()].double(), eps) * 0.5) < DT[dtype]
    none, _ = dec.parallel_step(x2, cols, 1.0, eps, ld=ld, n=3, dtype=dtype, mix=kw["mix"][:3], gates=gpad[:3, :ld].contiguous(), gate_b=kw["gate_b"],
                                x_out=x2, norm=False)
    want = table[ids.long()].double() + mix[:3].double() * ref.sigmoid(gates[:3, 0].double() + gb[0].double())
    assert none is None and _rel(x2[:, :cols], want) < (2e-6 if dtype == torch.float32 else 1e-5)


@pytest.mark.parametrize("t,e,k", [(1, 7, 3), (50, 10, 4), (333, 40, 33), (17, 130, 20), (9, 700, 8), (4, 1024, 40)])
def test_routing(t, e, k):
    from deepseek_v4_2080ti_b200.ops import moe
    gen = torch.Generator().manual_seed(e)
    z, corr = 2 * torch.randn(t, e + 5, generator=gen), 0.3 * torch.randn(e, generator=gen)
    idx, w = moe.route(z.cuda()[:, :e], corr.cuda(), k, "softmax", False, 1.0)
    want_i, want_w = ref.choose(z[:, :e].double(), corr.double(), k)
    assert torch.equal(idx.cpu().sort(-1).values.long(), want_i.sort(-1).values)
    s = torch.zeros(t, e).double().scatter_(1, idx.cpu().long(), w.double().cpu())
    assert _rel(s, torch.zeros(t, e).double().scatter_(1, want_i, want_w)) < 2e-6
    idx, w = moe.route(z.cuda()[:, :e], None, k, "sigmoid", True, 2.5)
    assert torch.allclose(w.sum(-1).cpu(), torch.full((t,), 2.5), rtol=1e-5)
    best = torch.sigmoid(z[:, :e]).topk(k).values
    assert torch.allclose(w.cpu() / w.cpu().sum(-1, keepdim=True), best / best.sum(-1, keepdim=True), rtol=1e-4)


@pytest.mark.parametrize("t,e,k,ident", [(1, 3, 2, 1), (40, 5, 4, 2), (700, 130, 6, 7), (5000, 9, 3, 0), (3, 1024, 8, 0)])
def test_plan_places_every_route_once(t, e, k, ident):
    from deepseek_v4_2080ti_b200.ops import _lib
    gen = torch.Generator().manual_seed(t)
    idx = torch.rand(t, e + ident, generator=gen).topk(min(k, e + ident)).indices.to(torch.int32)
    k, lo, r = idx.shape[1], 0, idx.numel()
    g = idx.cuda()
    i32 = lambda *s: torch.full(s, -7, dtype=torch.int32, device="cuda")
    off, row, tok, w1, w2, n1, n2 = i32(e + 1), i32(t, k), i32(r), i32(6 * (r + e), 4), i32(6 * (r + e), 4), i32(1), i32(1)
    rc = _lib.lib().b200_moe_plan(_lib.ptr(g), t, k, lo, e, _lib.ptr(off), _lib.ptr(row), _lib.ptr(tok), _lib.ptr(w1), _lib.ptr(n1), 3, 16, _lib.ptr(w2),
                                  _lib.ptr(n2), 2, 64, 6 * (r + e), _lib.stream())
    assert rc == 0
    cnt = torch.bincount(idx.flatten().long(), minlength=e + ident)[:e]
    want_off = torch.cat([torch.zeros(1, dtype=torch.long), cnt.cumsum(0)])
    assert torch.equal(off.cpu().long(), want_off)
    flat, nxt = row.cpu().flatten(), want_off[:-1].clone()
    for i, x in enumerate(idx.flatten().tolist()):
        if x >= e:
            assert flat[i] == -1
        else:                                                    # in order: results do not depend on the scheduling of blocks
            assert flat[i] == nxt[x] and int(tok[nxt[x]]) == i // k if i < 64 else flat[i] == nxt[x]
            nxt[x] += 1
    for work, num, mt, bn in ((w1, n1, 3, 16), (w2, n2, 2, 64)):
        rows = [(x, m, int(want_off[x]) + s, min(bn, int(cnt[x]) - s)) for x in range(e) for s in range(0, int(cnt[x]), bn) for m in range(mt)]
        assert int(num) == len(rows) and work[:len(rows)].cpu().tolist() == [list(v) for v in rows]


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("t,width,ff,e,ident,top,limit", [(1, 48, 20, 4, 2, 3, 0.9), (77, 100, 72, 6, 0, 2, 1.5), (600, 128, 64, 3, 1, 4, 0.5)])
def test_experts(dtype, t, width, ff, e, ident, top, limit):
    """Router, routed and shared experts of the runtime's own containers against the statement, summed by hand."""
    from deepseek_v4_2080ti_b200.ops import _lib, moe
    spec = kx.ExpertsSpec(ff, limit, e, ident, top, ff + 7, 2 * limit)
    cfg = kx.KemiraxConfig(32, width, 1e-5, [L(G(1, 16, 16, 4.0, 8), spec)])
    state = dict(kx.synth_state(cfg, 9))
    state["l0.mlp.router"] *= 4.0
    w = kx.KemiraxWeights(cfg, state, "cuda", dtype)
    rt = kx.KemiraxRuntime(cfg, w, max_context=64)
    h = torch.zeros(t, w.ld)
    h[:, :width] = torch.randn(t, width, generator=torch.Generator().manual_seed(t))
    h = h.to(dtype)
    out = rt._experts(w.layers[0].ff, h.cuda())
    _lib.check_status()
    sub = {n[len("l0.mlp."):]: v.double() for n, v in state.items() if n.startswith("l0.mlp.")}
    x = h[:, :width].double()
    z = moe.router_logits(h.cuda(), w.layers[0].ff.router)
    assert z.dtype == torch.float32 and _rel(z[:, :e + ident], x @ sub["router"].t()) < 3e-6
    r = out["routed"]
    got = torch.zeros(t, width).double()
    for i in range(t):
        for j in range(top):
            y = r.y[int(r.row[i, j]), :width].double().cpu() if int(r.idx[i, j]) < e else x[i]
            assert (int(r.row[i, j]) < 0) == (int(r.idx[i, j]) >= e)
            got[i] += float(r.weights[i, j]) * y
    got += ref.sigmoid(out["shared_gate"][:, :1].double().cpu()) * out["shared"][:, :width].double().cpu()
    mlp = cfg.to_json()["layers"][0]["mlp"]
    want = ref.experts(x, sub, mlp)
    err = (got - want).norm(dim=-1) / want.norm(dim=-1)
    assert float(err.max() if dtype == torch.float32 else err.median()) < DT[dtype]
