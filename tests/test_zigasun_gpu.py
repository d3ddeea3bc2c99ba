"""The Zigasun runtime on the GPU against the plain whole-sequence statement: prompts, token-by-token decoding, portions, mixed
batches, reused pages and state slots, long memories, and the public entry points; and the row kernels it shares."""
import random

import pytest
import torch

from deepseek_v4_2080ti_b200.models import zigasun as zg
from deepseek_v4_2080ti_b200.models.reference_cpu import zigasun_ref as ref

pytestmark = pytest.mark.gpu
F32_TOL = 3e-5
A, S, L = zg.AttentionSpec, zg.ScanSpec, zg.LayerSpec

CONFIGS = {
    # nothing is a multiple of anything; every kind of layer with and without a feed-forward; scan first
    "ragged": zg.ZigasunConfig(211, 84, 1e-3, 1.7, 0.8, [
        L(S(70, 10, 7, 4), 90, 1.2), L(A(6, 3, 20, 28, 0.3, 0.2, 0.4, 50)), L(S(52, 5, 30, 3)),
        L(A(3, 3, 20, 28, 0.25, 0.5, 0.2, 17, kv_from=1), 41, 0.6)]),
    # wide groups, values narrower than keys, one borrower right after the lender and one far behind
    "borrow": zg.ZigasunConfig(128, 128, 1e-6, 1.0, 1.0, [
        L(A(8, 1, 64, 32, 0.125, 0.1), 256, 4.0), L(A(8, 1, 64, 32, 0.1, 0.8, kv_from=0), 64, 1.0), L(S(128, 16, 8, 2), 64, 0.5),
        L(A(4, 1, 64, 32, 0.2, 0.3, 0.7, 9, kv_from=0))]),
    # attention only; values wider than one accumulator
    "wide": zg.ZigasunConfig(97, 64, 1e-5, 0.5, 1.3, [L(A(2, 1, 72, 144, 0.15, 0.25), 48, 2.0), L(A(4, 4, 16, 16, 0.3, 0.0))]),
    # scan only: no pages are ever read; one without a convolution history, one with a long one
    "scan": zg.ZigasunConfig(160, 96, 1e-5, 2.0, 0.5, [L(S(160, 32, 12, 1), 64, 1.0), L(S(96, 3, 5, 6)), L(S(48, 64, 16, 4), 160, 3.0)]),
}


class Case:
    """A runtime and the statement's logits for whole sequences (cached per sequence)."""

    def __init__(self, name, dtype, slots=4, context=512, blocks=None, block_size=64, poison=True, change=None):
        self.cfg, self.dtype = CONFIGS[name], dtype
        self.state = dict(zg.synth_state(self.cfg, seed=len(name)))
        if change:
            change(self.state)
        self.rt = zg.ZigasunRuntime(self.cfg, zg.ZigasunWeights(self.cfg, self.state, "cuda", dtype), max_slots=slots,
                                    max_context=context, num_blocks=blocks, block_size=block_size)
        if poison:                                   # what earlier requests may have left: nothing of it may show
            for i in range(len(self.cfg.layers)):
                if self.rt.k_cache[i] is not None:
                    self.rt.k_cache[i][1:] = 60.0
                    self.rt.v_cache[i][1:] = -90.0
                if self.rt.conv_tail[i] is not None:
                    self.rt.conv_tail[i].fill_(float("nan"))
                    self.rt.scan_state[i].fill_(float("nan"))
        self.raw, self.memo = self.cfg.to_json(), {}

    def want(self, toks):
        key = tuple(toks)
        if key not in self.memo:
            self.memo[key] = ref.forward(self.raw, self.state, toks, torch.float64)
        return self.memo[key]

    def near(self, got, want, tol=None):
        """Row errors relative to the spread of the logits.  In bf16 single rows can be ill-conditioned (a norm sits on the
        output of a sublayer that happens to cancel): one row in fifty may be off by more, no row by much."""
        d = got.double().cpu() - want
        d = d - d.mean(-1, keepdim=True)
        err = d.pow(2).mean(-1).sqrt() / want.std()
        if tol or self.dtype == torch.float32:
            assert float(err.max()) < (tol or F32_TOL), (float(err.max()), int(err.argmax()))
        else:
            over = int((err > 6e-2).sum())
            assert over <= max(1, err.numel() // 50) and float(err.max()) < 0.3 and float(err.mean()) < 4e-2, (over, float(err.max()), float(err.mean()))

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
        assert float((x.double() - y).norm() / y.norm()) < (3e-6 if dtype == torch.float32 else 3e-2)
    c.near(got, want)
    # with and without the tap: the same numbers (the update of the residual is only split in two launches)
    c.rt.free(slot)
    c.rt.residual_tap = None
    slot = c.rt.allocate()
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
def test_a_far_key_and_a_kept_first_token(dtype):
    """One loud early token: its key draws most of the attention of rows hundreds of positions away, and slow decays keep it in
    the scan's state.  Another early token gives other logits at the end; the runtime follows, in portions and decoding."""
    def change(state):
        state["l0.mix.A_log"] -= 5.0
        state["l0.mix.dt.b"] -= 2.0
        for n in ("l1.mix.q.norm", "l1.mix.k.norm"):
            state[n] *= 3.0
    c = Case("ragged", dtype, change=change)
    loud = c.state["embed"].float().norm(dim=-1).argmax().item()
    c.state["embed"][loud] *= 4.0
    c.rt.w.embed[loud] *= 4.0
    toks = [x if x != loud else (loud + 1) % c.cfg.vocab for x in _tokens(c.cfg, 330, seed=8)]
    with_it = [toks[0], loud] + toks[2:]
    w0, w1 = c.want(toks), c.want(with_it)
    assert float((w0[300:] - w1[300:]).pow(2).mean().sqrt() / w1.std()) > 0.15          # the far token shows
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
    c = Case("scan", dtype)
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
    cfg = CONFIGS["borrow"]
    zg.write_checkpoint(str(tmp_path), cfg, seed=4)
    prompts = [_tokens(cfg, n, seed=50 + n) for n in (45, 4, 18)]
    llm = LLM(EngineArgs(model=str(tmp_path), max_model_len=256, max_batch_size=3, dtype=dtype))
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=10))
    one = llm.generate([{"prompt_token_ids": prompts[0]}], SamplingParams(max_tokens=10))[0]
    if dtype == "float32":
        state = dict(zg.synth_state(cfg, 4))
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
    llm = LLM(EngineArgs(model="synthetic:zigasun-tiny", max_model_len=128, max_batch_size=2))
    assert len(llm.generate([{"prompt_token_ids": [1, 2, 3]}], SamplingParams(max_tokens=5))[0].token_ids) == 5
    llm.close()


def test_command_lines(tmp_path, capsys, monkeypatch):
    import io
    import json

    import numpy as np

    from deepseek_v4_2080ti_b200.cli import generate_gguf, trace_run
    cfg = CONFIGS["ragged"]
    zg.write_checkpoint(str(tmp_path / "m"), cfg, seed=2)
    state, raw = dict(zg.synth_state(cfg, 2)), cfg.to_json()
    toks = _tokens(cfg, 150, seed=61)
    want = ref.forward(raw, state, toks, torch.float64)
    assert generate_gguf.main(["--checkpoint", str(tmp_path / "m"), "--dtype", "float32", "--max-new-tokens", "1",
                               "--max-context", "256", "--token-ids", ",".join(map(str, toks))]) == 0
    out = capsys.readouterr().out
    assert f"tokens={int(want[-1].argmax())}\n" in out and "family=zigasun" in out
    (tmp_path / "o").mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:100], "want": [99, 0]}, {"id": "y", "tokens": toks[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[1:2], "want": [0]}, {"id": "x", "tokens": toks[100:], "want": [49]}], "end": ["y", "x"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert trace_run.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "256"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1"]
    for n, places in ((0, [99, 0]), (1, [1, 149])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", dtype="<f4").copy()).view(2, cfg.vocab).double()
        assert float((got - want[places]).abs().max() / want.std()) < 1e-4


# ---------------------------------------------------------------------------------------------- shared row kernels
DT = {torch.bfloat16: 1.2e-2, torch.float32: 2e-6}


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-30))


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("cols", [20, 333, 4096])
def test_residual_boundary_without_an_input_norm(dtype, cols):
    """A scaled embedding row starts the residual, the sublayer's output enters through its norm, and the next sublayer reads
    the residual itself."""
    from deepseek_v4_2080ti_b200.ops import decoder as dec
    gen = torch.Generator().manual_seed(cols)
    ld, eps = dec.pad16(cols), 1e-3
    pad = lambda t, dt: torch.nn.functional.pad(t, (0, ld - cols)).to("cuda", dt).contiguous()
    table, d, w = (torch.randn(*s, generator=gen) for s in ((9, cols), (4, cols), (cols,)))
    table, d = table.to(dtype), d.to(dtype)
    ids = torch.tensor([8, 0, 3, 3], dtype=torch.int32)
    x = torch.full((4, ld), 5.0).cuda()
    y = dec.residual_norm(x, cols, eps, ids=ids.cuda(), table=pad(table, dtype), table_scale=3.7, rms=True, plain=True)
    want = table[ids.long()].double() * 3.7
    assert _rel(x[:, :cols], want) < 1e-6 and _rel(y[:, :cols], want) < DT[dtype] and not x[:, cols:].any()
    y = dec.residual_norm(x, cols, eps, delta=pad(d, dtype), post_w=pad(0.4 * w, torch.float32), rms=True, plain=True)
    want = want + 0.4 * ref.rms(d.double(), eps) * w.double()
    assert y.dtype == dtype and _rel(x[:, :cols], want) < 2e-6 and _rel(y[:, :cols], want) < DT[dtype]
    assert ld == cols or not y[:, cols:].any()


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("t,width,ff,limit", [(5, 48, 70, 0.9), (300, 64, 128, 2.0), (512, 192, 256, 1.0), (256, 128, 640, 0.3)])
def test_gated_unit(dtype, t, width, ff, limit):
    """Both forms: in the epilogue of the pair GEMM (evenly tiled bf16 batches) and as a kernel of its own."""
    from deepseek_v4_2080ti_b200.ops import _lib, decoder as dec, gemm
    gen = torch.Generator().manual_seed(ff)
    g, u, x = (torch.randn(*s, generator=gen).to(torch.bfloat16) for s in ((ff, width), (ff, width), (t, width)))
    g, u = g * 0.3, u * 0.3
    p = dec.Projection.make(dec.interleave_glu(g, u), dtype, "cuda")
    if dtype == torch.bfloat16 and t % 256 == 0 and width % 64 == 0:
        assert gemm.glu_fusable(t, p.packed)
    got = p.glu(x.to("cuda", dtype), limit)
    _lib.check_status()
    eye = torch.eye(ff).double()
    want = ref.clamped_glu(x.double(), {"gate": g.double(), "up": u.double(), "down": eye}, limit)
    assert _rel(got[:, :ff], want) < DT[dtype] and not got[:, ff:].any()
    # without a limit: the plain unit
    plain = p.glu(x.to("cuda", dtype), 0.0)
    a, b = x.double() @ g.double().t(), x.double() @ u.double().t()
    assert _rel(plain[:, :ff], ref.silu(a) * b) < DT[dtype]
