"""The Rutulix runtime on the GPU against the plain whole-sequence statement: prompts, token-by-token decoding, portions,
mixed batches, reused pages and slots, chunk and page borders, long decoding, and the public entry points."""
import random

import pytest
import torch

from deepseek_v4_2080ti_b200.models import rutulix as rx
from deepseek_v4_2080ti_b200.models.reference_cpu import rutulix_ref as ref

pytestmark = pytest.mark.gpu
F32_TOL = 2e-5


def _spec(heads, kv, dim, chunk, rot, scale, base=400.0, scaling=None):
    return rx.AttentionSpec(heads, kv, dim, scale, chunk, rot, base, scaling)


Y = {"factor": 3.0, "original": 96, "fast": 12.0, "slow": 1.0}
CONFIGS = {
    # layers that differ in everything, one without a feed-forward, sizes that are multiples of nothing, a loop at the start
    "ragged": rx.RutulixConfig(211, 84, 1e-3, [
        rx.LayerSpec(_spec(6, 3, 20, 29, 12, 0.21, scaling=Y), 90), rx.LayerSpec(_spec(3, 1, 24, 50, 24, 0.3), 0),
        rx.LayerSpec(_spec(5, 5, 10, 64, 2, 0.4, 30.0, dict(Y, factor=1.0)), 41)], (0, 2, 3)),
    # one pass of the loop still adds its step; loop in the middle; wide groups
    "once": rx.RutulixConfig(128, 128, 1e-6, [
        rx.LayerSpec(_spec(8, 1, 16, 40, 16, 0.25, scaling=Y), 256), rx.LayerSpec(_spec(4, 2, 64, 40, 32, 0.1, 5000.0), 64),
        rx.LayerSpec(_spec(8, 2, 16, 33, 8, 0.25), 128)], (1, 2, 1)),
    # no loop; one layer looks at everything, so nothing may be given back early
    "open": rx.RutulixConfig(97, 64, 1e-5, [rx.LayerSpec(_spec(4, 4, 16, 0, 8, 0.25, scaling=Y), 48),
                                            rx.LayerSpec(_spec(2, 1, 40, 17, 40, 0.2), 0)], None),
    # the loop reaches the last layer
    "tail": rx.RutulixConfig(160, 96, 1e-5, [rx.LayerSpec(_spec(2, 2, 32, 100, 16, 0.2, scaling=Y), 64),
                                             rx.LayerSpec(_spec(6, 2, 32, 100, 16, 0.2, scaling=Y), 160)], (1, 2, 4)),
}


class Case:
    """A runtime and the statement's logits for whole sequences (cached per sequence)."""

    def __init__(self, name, dtype, slots=4, context=512, blocks=None, block_size=64):
        self.cfg, self.dtype = CONFIGS[name], dtype
        self.state = dict(rx.synth_state(self.cfg, seed=len(name)))
        w = rx.RutulixWeights(self.cfg, self.state, "cuda", dtype)
        self.rt = rx.RutulixRuntime(self.cfg, w, max_slots=slots, max_context=context, num_blocks=blocks, block_size=block_size)
        self.raw, self.memo = self.cfg.to_json(), {}

    def want(self, toks):
        key = tuple(toks)
        if key not in self.memo:
            self.memo[key] = ref.forward(self.raw, self.state, toks, torch.float64)
        return self.memo[key]

    def near(self, got, want, tol=None):
        """Worst row error, relative to the spread of the logits."""
        d = got.double().cpu() - want
        d = d - d.mean(-1, keepdim=True)
        err = float((d.pow(2).mean(-1).sqrt() / want.std()).max())
        limit = tol or (F32_TOL if self.dtype == torch.float32 else 3e-2)
        assert err < limit, err

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
    c.rt.residual_tap = lambda run, x: taps.append((run, x.cpu()))
    slot = c.rt.allocate()
    got = c.rt.step([(slot, toks, list(range(203)))])
    _lib.check_status()
    want = ref.forward(c.raw, c.state, toks, torch.float64, want_taps)
    assert [r for r, _ in taps] == list(range(len(c.cfg.runs())))
    for (_, x), y in zip(taps, want_taps):
        assert float((x.double() - y).norm() / y.norm()) < (2e-6 if dtype == torch.float32 else 1.5e-2)
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
    # prompt first, then decoding across chunk and page borders
    slot = c.rt.allocate()
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


def test_first_tokens_and_single_token_requests():
    c = Case("once", torch.float32)
    for n in (1, 2, 3):
        toks = _tokens(c.cfg, n, seed=30 + n)
        slot = c.rt.allocate()
        c.near(c.rt.step([(slot, toks, list(range(n)))]), c.want(toks))
        c.rt.free(slot)


@BOTH
def test_long_decoding_gives_pages_back(dtype):
    c = Case("ragged", dtype, slots=1, context=512, blocks=5)           # 4 pages for a sequence of 7
    toks = _tokens(c.cfg, 420, seed=5)
    slot = c.rt.allocate()
    got = c.feed(slot, toks, [40] + [1] * 380)
    assert c.rt.seqs[slot].retired >= 5
    c.near(got, c.want(toks))
    c.rt.free(slot)
    assert len(c.rt.free_blocks) == 4


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


def _alone(c, prompt, n):
    return c.rt.generate(torch.tensor(prompt, dtype=torch.int32), n)


def test_scheduler_batches_match_each_request_alone():
    from deepseek_v4_2080ti_b200.runtime.step_scheduler import StepScheduler
    c = Case("tail", torch.float32, slots=3, context=256, blocks=10)
    reqs = [(_tokens(c.cfg, n, seed=40 + n), m) for n, m in ((70, 12), (3, 40), (1, 25), (120, 9), (20, 20), (64, 64))]
    sched = StepScheduler(c.rt, (), max_batch=3, token_budget=48)
    for i, (p, m) in enumerate(reqs):
        sched.submit(i, p, m)
    res = sched.run()
    assert sched.mixed_rounds > 0
    for i, (p, m) in enumerate(reqs):
        assert res[i][0] == _alone(c, p, m), i


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_public_api_serves_a_checkpoint_folder(tmp_path, dtype):
    from pocketllm import LLM, EngineArgs, SamplingParams
    cfg = CONFIGS["once"]
    rx.write_checkpoint(str(tmp_path), cfg, seed=4)
    prompts = [_tokens(cfg, n, seed=50 + n) for n in (45, 4, 18)]
    llm = LLM(EngineArgs(model=str(tmp_path), max_model_len=256, max_batch_size=3, dtype=dtype))
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=10))
    one = llm.generate([{"prompt_token_ids": prompts[0]}], SamplingParams(max_tokens=10))[0]
    if dtype == "float32":
        state = dict(rx.synth_state(cfg, 4))
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


def test_command_lines(tmp_path, capsys, monkeypatch):
    import io
    import json

    import numpy as np

    from deepseek_v4_2080ti_b200.cli import generate_gguf, trace_run
    cfg = CONFIGS["tail"]
    rx.write_checkpoint(str(tmp_path / "m"), cfg, seed=2)
    state, raw = dict(rx.synth_state(cfg, 2)), cfg.to_json()
    toks = _tokens(cfg, 150, seed=61)
    want = ref.forward(raw, state, toks, torch.float64)
    assert generate_gguf.main(["--checkpoint", str(tmp_path / "m"), "--dtype", "float32", "--max-new-tokens", "1",
                               "--max-context", "256", "--token-ids", ",".join(map(str, toks))]) == 0
    out = capsys.readouterr().out
    assert f"tokens={int(want[-1].argmax())}\n" in out and "family=rutulix" in out
    (tmp_path / "o").mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:100], "want": [99, 0]}, {"id": "y", "tokens": toks[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[1:2], "want": [0]}, {"id": "x", "tokens": toks[100:], "want": [49]}], "end": ["y", "x"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert trace_run.main(["--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "256"]) == 0
    assert capsys.readouterr().out.split() == ["done", "0", "done", "1"]
    for n, places in ((0, [99, 0]), (1, [1, 149])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", dtype="<f4").copy()).view(2, cfg.vocab).double()
        assert float((got - want[places]).abs().max() / want.std()) < 1e-4


def test_gqa_family_runs_mixed_steps():
    """The mixed-batch step is the shared runtime's: the GGUF GQA family runs portions beside single tokens as well."""
    from deepseek_v4_2080ti_b200.models import gqa_moe as gm
    cfg = gm.GqaMoeConfig.tiny(layers=2, experts=8)
    cfg.attn_type = cfg.dense_type = "Q8_0"
    cfg.gate_up_type, cfg.down_type = "Q2_K", "Q2_K"
    store = gm.TensorStore(list(gm.synth_tensors(cfg, seed=5, device="cuda", std=0.05)))
    rt = gm.GqaMoeRuntime(cfg, gm.GqaMoeGpuWeights(cfg, store, "cuda"), max_slots=2, max_context=256)
    tensors = {k: v.cpu() for k, v in store.dequantized().items()}
    a, b = _tokens(cfg, 60, seed=1), _tokens(cfg, 75, seed=2)
    wa, wb = (gm.GqaMoeReference(cfg, tensors).forward(torch.tensor(x)) for x in (a, b))
    sa, sb = rt.allocate(), rt.allocate()
    rt.step([(sa, a[:50], [])])
    got = rt.step([(sa, a[50:51], [0]), (sb, b[:70], [69])])
    got2 = rt.step([(sb, b[70:], [4]), (sa, a[51:52], [0])])
    for g, w in ((got[0], wa[50]), (got[1], wb[69]), (got2[0], wb[74]), (got2[1], wa[51])):
        assert float((g.cpu() - w).norm() / w.norm()) < 0.08
