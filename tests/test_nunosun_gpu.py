"""The Nunosun runtime on the GPU against the plain whole-sequence statement: prompts, token-by-token decoding, portions, mixed
batches, reused pages and state slots, keys at the windows' edges and long memories, and the public entry points; and the
residual step, the activations, the routing and the expert kernels it uses."""
import math
import random

import pytest
import torch

from deepseek_v4_2080ti_b200.models import nunosun as ns
from deepseek_v4_2080ti_b200.models.reference_cpu import nunosun_ref as ref

pytestmark = pytest.mark.gpu
F32_TOL = 4e-5
W, R, P, D, F, E, L = ns.WindowSpec, ns.RetentionSpec, ns.PairSpec, ns.DeltaSpec, ns.DenseSpec, ns.ExpertsSpec, ns.LayerSpec

CONFIGS = {
    # nothing is a multiple of anything; every mixer with every feed-forward and without one, windows and tables that differ
    "ragged": ns.NunosunConfig(211, 84, 1e-3, 13, 3, 0.7, [
        L(D(4, 2, 20, 28, 4), F(90)), L(P(W(6, 3, 20, 12, 0.3, 37, 90, 14), R(3, 18, 28, (0.7, 0.97, 0.999), 10, 300.0)), E(22, 5, 2)),
        L(D(3, 3, 12, 44, 2)), L(P(W(2, 1, 36, 60, 0.2, 75, 40, 9), R(2, 36, 10, (0.9, 0.995), 36, 5000.0)), F(41)),
        L(D(5, 1, 33, 17, 1), E(30, 3, 3)), L(P(W(3, 3, 16, 16, 0.25, 1, 8, 4), R(1, 20, 50, (0.98,), 4, 50.0)))]),
    # sizes the tensor-core kernels tile evenly; a window longer than any sequence beside a short one
    "even": ns.NunosunConfig(128, 128, 1e-6, 32, 4, 2.0, [
        L(P(W(4, 2, 64, 64, 0.125, 1000, 256, 32), R(2, 64, 64, (0.96, 0.998), 64, 10000.0)), E(64, 8, 3)), L(D(4, 2, 64, 64, 4), F(256)),
        L(P(W(2, 2, 128, 128, 0.1, 64, 128, 16), R(2, 128, 64, (0.99, 0.9), 64, 10000.0)), F(192)), L(D(2, 2, 128, 128, 3), E(32, 4, 1))]),
    # attention heads wider than the tile kernel takes; no convolution over rows; one expert of one
    "wide": ns.NunosunConfig(97, 64, 1e-5, 8, 1, 1.0, [
        L(P(W(2, 1, 208, 272, 0.07, 50, 30, 12), R(2, 160, 80, (0.95, 0.99), 160, 1000.0)), E(48, 1, 1)), L(D(2, 1, 160, 96, 5), F(64))]),
    # recurrent only: no pages are ever read
    "recurrent": ns.NunosunConfig(160, 96, 1e-5, 24, 6, 0.5, [L(D(2, 1, 64, 64, 3), F(80)), L(D(4, 4, 16, 32, 4), E(40, 6, 4)), L(D(1, 1, 32, 16, 2))]),
}


class Case:
    def __init__(self, name, dtype, slots=3, context=512, blocks=None, block_size=64, change=None):
        self.cfg, self.dtype = CONFIGS[name], dtype
        self.state = dict(ns.synth_state(self.cfg, seed=len(name)))
        if change:
            change(self.state)
        self.rt = ns.NunosunRuntime(self.cfg, ns.NunosunWeights(self.cfg, self.state, "cuda", dtype), max_slots=slots,
                                    max_context=context, num_blocks=blocks, block_size=block_size)
        for i in range(len(self.cfg.layers)):        # what earlier requests may have left: nothing of it may show
            for t in (self.rt.k_cache[i], self.rt.v_cache[i]):
                if t is not None:
                    t[1:] = 60.0
            for t in (self.rt.state[i], self.rt.row_tail[i], self.rt.conv_tail[i]):
                if t is not None:
                    t.fill_(float("nan"))
        self.raw, self.memo = self.cfg.to_json(), {}

    def want(self, toks):
        key = tuple(toks)
        if key not in self.memo:
            self.memo[key] = ref.forward(self.raw, self.state, toks, torch.float64)
        return self.memo[key]

    def near(self, got, want, tol=None):
        """Row errors relative to the spread of the logits.  In bf16 a token may choose another expert where two logits are
        equal within rounding: a few rows may be off by more."""
        d = got.double().cpu() - want
        d = d - d.mean(-1, keepdim=True)
        err = d.pow(2).mean(-1).sqrt() / want.std()
        if tol or self.dtype == torch.float32:
            assert float(err.max()) < (tol or F32_TOL), (float(err.max()), int(err.argmax()))
        else:
            over = int((err > 7e-2).sum())
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
    for n in (1, 2, 3, 5):
        toks = _tokens(c.cfg, n, seed=30 + n)
        for cuts in ([n], [1] * n):
            slot = c.rt.allocate()
            c.near(c.feed(slot, toks, cuts), c.want(toks))
            c.rt.free(slot)


@BOTH
def test_long_decoding_gives_pages_back(dtype):
    c = Case("ragged", dtype, slots=1, context=512, blocks=5, block_size=32)      # 16 pages would hold the sequence
    toks = _tokens(c.cfg, 420, seed=5)
    slot = c.rt.allocate()
    c.near(c.feed(slot, toks, [40] + [1] * 380), c.want(toks))
    assert c.rt.history_span() == 74 and len(c.rt.free_blocks) >= 0 and sum(b != 0 for b in c.rt.seqs[slot].blocks) <= 4


@BOTH
@pytest.mark.parametrize("how", ["prompt", "portions", "decoding"])
def test_window_edges_show(dtype, how):
    """Flat attention (no query stands out) with everything else that mixes rows silenced: another token shows in the logits of
    the last position that sees it, and the position behind has nothing of it."""
    size = 64

    def change(state):
        for n in state:
            if n.endswith(("right.out", "canon1")) or n == "l0.mix.left.out" or (n.startswith(("l1.", "l3.")) and n.endswith(".mix.o")):
                state[n] = torch.zeros_like(state[n])
        state["l2.mix.left.q.norm"] = torch.zeros_like(state["l2.mix.left.q.norm"])
    c = Case("even", dtype, change=change)
    toks = _tokens(c.cfg, 200, seed=8)
    with_it = list(toks)
    with_it[70] = (toks[70] + 5) % c.cfg.vocab
    w0, w1 = c.want(toks), c.want(with_it)
    diff = (w0 - w1).pow(2).mean(-1).sqrt() / w1.std()
    inside, outside = 70 + size - 1, 70 + size
    assert float(diff[inside]) > 1e-3 and float(diff[outside:].max()) < 1e-9
    cuts = {"prompt": [200], "portions": [69, 2, 62, 2, 65], "decoding": [60] + [1] * 140}[how]
    got = []
    for s in (toks, with_it):
        slot = c.rt.allocate()
        got.append(c.feed(slot, s, cuts))
        c.near(got[-1], w1 if s is with_it else w0)
        c.rt.free(slot)
    shows = (got[0] - got[1]).double().cpu().pow(2).mean(-1).sqrt() / w1.std()
    assert float(shows[inside]) > 0.5 * float(diff[inside]) and float(shows[outside:].max()) < 1e-6


@BOTH
def test_a_far_token_shows(dtype):
    """Slow decays: another token far outside every window gives other logits hundreds of positions later, and the runtime
    follows, in one portion, in several and decoding."""
    def change(state):
        for i in (0, 2, 4):
            state[f"l{i}.mix.A_log"] = torch.full_like(state[f"l{i}.mix.A_log"], -6.0)
            state[f"l{i}.mix.dt_bias"] = torch.full_like(state[f"l{i}.mix.dt_bias"], -4.0)
            state[f"l{i}.mix.b"] *= 0.2
    c = Case("ragged", dtype, change=change)
    loud = c.state["embed"].float().norm(dim=-1).argmax().item()
    toks = [x if x != loud else (loud + 1) % c.cfg.vocab for x in _tokens(c.cfg, 330, seed=8)]
    with_it = [toks[0], loud] + toks[2:]
    w0, w1 = c.want(toks), c.want(with_it)
    assert float((w0[300:] - w1[300:]).pow(2).mean().sqrt() / w1.std()) > 1e-3          # the far token shows
    for cuts in ([330], [70, 2, 1, 1, 200, 56], [290] + [1] * 40):
        got = []
        for s, w in ((toks, w0), (with_it, w1)):
            slot = c.rt.allocate()
            got.append(c.feed(slot, s, cuts))
            c.near(got[-1], w)
            c.rt.free(slot)
        if dtype == torch.float32:
            c.near(got[1] - got[0] + w0.float().cuda(), w1)


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
    ns.write_checkpoint(str(tmp_path), cfg, seed=4)
    prompts = [_tokens(cfg, n, seed=50 + n) for n in (45, 4, 18)]
    llm = LLM(EngineArgs(model=str(tmp_path), max_model_len=256, max_batch_size=3, dtype=dtype))
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=10))
    one = llm.generate([{"prompt_token_ids": prompts[0]}], SamplingParams(max_tokens=10))[0]
    if dtype == "float32":
        state = dict(ns.synth_state(cfg, 4))
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
    llm = LLM(EngineArgs(model="synthetic:nunosun-tiny", max_model_len=128, max_batch_size=2))
    assert len(llm.generate([{"prompt_token_ids": [1, 2, 3]}], SamplingParams(max_tokens=5))[0].token_ids) == 5
    llm.close()


def test_command_lines(tmp_path, capsys, monkeypatch):
    import io
    import json

    import numpy as np

    from deepseek_v4_2080ti_b200.cli import generate_gguf, trace_run
    cfg = CONFIGS["ragged"]
    ns.write_checkpoint(str(tmp_path / "m"), cfg, seed=2)
    state, raw = dict(ns.synth_state(cfg, 2)), cfg.to_json()
    toks = _tokens(cfg, 150, seed=61)
    want = ref.forward(raw, state, toks, torch.float64)
    assert generate_gguf.main(["--checkpoint", str(tmp_path / "m"), "--dtype", "float32", "--max-new-tokens", "1",
                               "--max-context", "256", "--token-ids", ",".join(map(str, toks))]) == 0
    out = capsys.readouterr().out
    assert f"tokens={int(want[-1].argmax())}\n" in out and "family=nunosun" in out
    (tmp_path / "o").mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:100], "want": [99, 0]}, {"id": "y", "tokens": toks[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[1:2], "want": [0]}, {"id": "x", "tokens": toks[100:], "want": [49]}], "end": ["y", "x"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert trace_run.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "256"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1"]
    for n, places in ((0, [99, 0]), (1, [1, 149])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", dtype="<f4").copy()).view(2, cfg.vocab).double()
        assert float((got - want[places]).abs().max() / want.std()) < 2e-4


# ---------------------------------------------------------------------------------------------- residual step, activations, experts
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
@pytest.mark.parametrize("cols,single,taps", [(20, True, 4), (333, False, 3), (4112, True, 2), (4112, False, 7), (9000, False, 1), (60, True, 1)])
def test_residual_step(dtype, cols, single, taps):
    """Everything the residual takes at once, the norm, and the convolution of its rows across portions and slots."""
    from deepseek_v4_2080ti_b200.ops import decoder as dec
    entries = [(2, 1), (0, 1), (4, 1)] if single else [(2, 5), (0, 1), (4, 2), (1, 9)]
    pos0 = {2: 7, 0: 0, 4: 2, 1: 0}
    n, ld, eps, top, keep = sum(k for _, k in entries), dec.pad16(cols), 1e-3, 5, taps - 1
    gen = torch.Generator().manual_seed(cols)
    r = lambda *s: torch.randn(*s, generator=gen)
    pad = lambda t, dt: torch.nn.functional.pad(t, (0, ld - t.shape[-1])).to("cuda", dt).contiguous()
    x, a, b, p0, p1 = r(n, cols), *(r(n, cols).to(dtype) for _ in range(4))
    wa, wb, wn, cw = r(cols), r(cols), r(cols), r(taps, cols)
    wts, row = torch.rand(n, top, generator=gen), torch.randperm(n * top, generator=gen).to(torch.int32).view(n, top)
    row[0, 1] = -1
    y, tail = r(n * top, cols).to(dtype), r(5, max(keep, 1), cols).to(dtype)
    want_x = x.double() + ref.rms(a.double(), eps) * wa + ref.rms(b.double(), eps) * wb + p0.double() + p1.double()
    for t in range(n):
        for k in range(top):
            if row[t, k] >= 0:
                want_x[t] += wts[t, k].double() * y[row[t, k]].double()
    want_h = ref.rms(want_x, eps) * wn
    f32 = lambda t: pad(t, torch.float32)
    xg, tg = f32(x), pad(tail, dtype)
    pos = torch.tensor([pos0[s] + j for s, k in entries for j in range(k)], dtype=torch.int32).cuda()
    cg = f32(cw)
    cg[-1, :cols] += 1.0
    routed = dec.Routed(torch.nn.functional.pad(pad(y, dtype), (0, 16)), row.cuda(), row.cuda(), wts.cuda(), 1)
    kw = dict(ld=ld, n=n, dtype=dtype, normed=((pad(a, dtype), f32(wa)), (pad(b, dtype), f32(wb))), plain=(pad(p0, dtype), pad(p1, dtype)),
              routed=routed, weight=f32(wn))
    pick = torch.tensor([n - 1, 0], dtype=torch.int32).cuda()
    none, some, no_m = dec.branch_step(xg, cols, eps, **kw, rows=pick)
    assert none is None and no_m is None and _rel(some[:, :cols], want_h[[n - 1, 0]]) < DT[dtype] and torch.equal(xg, f32(x))
    cp, hg, mg = dec.branch_step(xg, cols, eps, **kw, x_out=xg, copy=True, conv=cg, tail=tg, seg=_segments(entries), positions=pos)
    assert _rel(xg[:, :cols], want_x) < (2e-6 if dtype == torch.float32 else 1e-5) and not xg[:, cols:].any()
    assert torch.equal(cp, xg.to(dtype)) and _rel(hg[:, :cols], want_h) < DT[dtype] and not hg[:, cols:].any() and not mg[:, cols:].any()
    hq, at = hg[:, :cols].double().cpu(), 0                           # the convolution works on the rounded norm
    for s, k in entries:
        before = tail[s].double().clone()
        for j in range(max(keep, 1)):
            if keep - j > pos0[s]:
                before[j] = 0.0                                        # nothing before the sequence, whatever the slot holds
        full = torch.cat([before[:keep], hq[at:at + k]])
        for t in range(k):
            want_m = hq[at + t] + sum(cw[j].double() * full[t + j] for j in range(taps))
            assert _rel(mg[at + t, :cols], want_m) < DT[dtype], (s, t)
        if keep:
            kept = tg[s, :, :cols].double().cpu()
            for j in range(keep):
                if keep - j <= pos0[s] + k:
                    assert torch.equal(kept[j], full[k + j]), (s, j)
        at += k
    assert torch.equal(tg[3, :, :cols].cpu(), tail[3])                 # nobody's slot
    # an embedding row behind its norm as the start, and a step without a norm
    table, ids = r(9, cols).to(dtype), torch.tensor([8, 0, 3], dtype=torch.int32)
    x2 = torch.full((3, ld), 5.0).cuda()
    _, h2, _ = dec.branch_step(None, cols, eps, ld=ld, n=3, dtype=dtype, ids=ids.cuda(), table=pad(table, dtype), normed=((None, f32(wa)),), x_out=x2,
                               weight=f32(wn))
    start = ref.rms(table[ids.long()].double(), eps) * wa
    assert _rel(x2[:, :cols], start) < 2e-6 and _rel(h2[:, :cols], ref.rms(start, eps) * wn) < DT[dtype]
    none, no_h, _ = dec.branch_step(x2, cols, eps, ld=ld, n=3, dtype=dtype, plain=(pad(p0[:3], dtype),), x_out=x2)
    assert none is None and no_h is None and _rel(x2[:, :cols], start + p0[:3].double()) < 2e-6


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("cols", [1, 24, 90, 2000, 3111, 8448, 20000])
def test_polynomial_of_row_norms(dtype, cols):
    from deepseek_v4_2080ti_b200.ops import decoder as dec
    ld = dec.pad16(cols)
    z = torch.randn(7, cols, generator=torch.Generator().manual_seed(cols)).to(dtype)
    z[3] *= 30.0
    z[4] *= 0.01
    full = torch.full((7, ld + 32), 9.0, dtype=dtype)
    full[:, :cols] = z
    coef = (0.7, -0.4, 0.3, 0.15)
    got = dec.poly_norm(full.cuda(), cols, coef, 1e-5, ld)
    want = ref.poly_norm(z.double(), torch.tensor(coef).double(), 1e-5)
    assert got.shape == (7, ld) and not got[:, cols:].any()
    for i in range(7):
        assert _rel(got[i, :cols], want[i]) < DT[dtype], i


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("t,width,side", [(1, 84, 13), (33, 2048, 256), (64, 100, 16), (65, 100, 48), (300, 128, 8)])
def test_token_gate(dtype, t, width, side):
    from deepseek_v4_2080ti_b200.ops import decoder as dec
    gen = torch.Generator().manual_seed(t)
    w, x = torch.randn(side, width, generator=gen).bfloat16() * (4 / width ** 0.5), torch.randn(t, width, generator=gen).to(dtype)
    sp, ld = dec.pad16(side), dec.pad16(width)
    table = torch.zeros(50, 3, sp)
    table[:, :, :side] = torch.randn(50, 3, side, generator=gen)
    table = table.to(dtype)
    ids = torch.randint(0, 50, (t,), generator=gen, dtype=torch.int32)
    proj = dec.Projection.make(w, dtype, "cuda")
    got = dec.token_gate(torch.nn.functional.pad(x, (0, ld - width)).cuda(), proj, table.view(50, -1).cuda(), 2 * sp, ids.cuda())
    want = ref.gelu_tanh(x.double() @ w.double().t()) * table[ids.long(), 2, :side].double()
    assert _rel(got[:, :side], want) < DT[dtype] and not got[:, side:].any()


@pytest.mark.parametrize("t,e,k", [(1, 7, 3), (50, 10, 4), (333, 40, 33), (17, 130, 20), (9, 700, 8), (4, 1024, 40), (6, 1, 1)])
def test_routing_by_the_chosen_logits(t, e, k):
    from deepseek_v4_2080ti_b200.ops import moe
    gen = torch.Generator().manual_seed(e)
    z, bias = 6 * torch.randn(t, e + 5, generator=gen), 2.0 * torch.randn(e, generator=gen)
    idx, w = moe.route(z.cuda()[:, :e], bias.cuda(), k, "softmax_chosen", True, 1.0)
    want_i, want_w = ref.choose(z[:, :e].double() + bias.double(), k)
    assert torch.equal(idx.cpu().long(), want_i)                       # largest first
    assert _rel(w, want_w) < 2e-6 and torch.allclose(w.sum(-1).cpu(), torch.ones(t), atol=1e-5)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("t,width,ff,e,top", [(1, 48, 20, 4, 3), (77, 100, 72, 6, 2), (600, 128, 64, 3, 1)])
def test_experts(dtype, t, width, ff, e, top):
    from deepseek_v4_2080ti_b200.ops import _lib
    cfg = ns.NunosunConfig(32, width, 1e-5, 8, 2, 1.0, [L(D(1, 1, 16, 16, 2), E(ff, e, top))])
    state = dict(ns.synth_state(cfg, 9))
    state["l0.mlp.router"] *= 4.0
    w = ns.NunosunWeights(cfg, state, "cuda", dtype)
    rt = ns.NunosunRuntime(cfg, w, max_context=64)
    h = torch.zeros(t, w.ld)
    h[:, :width] = torch.randn(t, width, generator=torch.Generator().manual_seed(t))
    h = h.to(dtype)
    r = rt._experts(w.layers[0].ff, h.cuda())
    _lib.check_status()
    sub = {n[len("l0.mlp."):]: v.double() for n, v in state.items() if n.startswith("l0.mlp.")}
    got = torch.zeros(t, width).double()
    for i in range(t):
        for j in range(top):
            got[i] += float(r.weights[i, j]) * r.y[int(r.row[i, j]), :width].double().cpu()
    want = ref.experts(h[:, :width].double(), sub, cfg.to_json()["layers"][0]["mlp"])
    err = (got - want).norm(dim=-1) / want.norm(dim=-1)
    assert float(err.max() if dtype == torch.float32 else err.median()) < DT[dtype]
    assert math.isfinite(float(err.max()))
