"""Kemirax decoder on the CPU: configuration and tensor inventory, registry, the plain statement's own invariants, and the
weight layouts of the serving path against it."""
import math

import pytest
import torch

from deepseek_v4_2080ti_b200.models import kemirax as kx, registry
from deepseek_v4_2080ti_b200.models.reference_cpu import kemirax_ref as ref
from deepseek_v4_2080ti_b200.ops import decoder, mixattn

YARN = {"factor": 3.0, "original": 64, "fast": 4.0, "slow": 0.5}


def _cfg():
    return kx.KemiraxConfig(61, 36, 1e-4, [
        kx.LayerSpec(kx.LinearSpec(3, 10, 14, 5.0, rank=6), kx.ExpertsSpec(22, 1.5, 5, 2, 3, 30, 0.8)),
        kx.LayerSpec(kx.LatentSpec(5, 12, 6, 18, 20, 28, 0.3, 6, 500.0, YARN)),
        kx.LayerSpec(kx.LatentSpec(2, 7, 6, 9, 11, 28, 0.2, 6, 500.0, YARN, kv_from=1), kx.ExpertsSpec(9, 0.7, 3, 0, 1)),
        kx.LayerSpec(kx.LinearSpec(1, 24, 5, 1.0, rank=20), kx.ExpertsSpec(16, 2.0, 1, 1, 2, 8, 3.0))])


def test_config_round_trip_and_inventory():
    cfg = _cfg()
    assert kx.KemiraxConfig.from_json(cfg.to_json()) == cfg and cfg.vocab_size == 61
    s = cfg.tensor_shapes()
    assert s["l0.mix.q"] == (30, 36) and s["l0.mix.v"] == s["l0.mix.g"] == (42, 36) and s["l0.mix.a2"] == (30, 6) and s["l0.mix.norm"] == (14,)
    assert s["l0.mlp.e4.down"] == (36, 22) and "l0.mlp.e5.up" not in s and s["l0.mlp.router"] == (7, 36) and s["l0.mlp.shared.sg"] == (1, 36)
    assert s["l1.mix.uq"] == (90, 20) and s["l1.mix.dkv"] == (34, 36) and s["l1.mix.uv"] == (90, 28) and s["l1.mix.o"] == (36, 90)
    assert "l1.rg2" not in s and "l1.mlp.router" not in s and s["l1.rg1"] == (36, 36) and s["l1.norm1"] == s["final.norm"] == ()
    assert "l2.mix.dkv" not in s and "l2.mix.dkv.norm" not in s and s["l2.mix.uk"] == (14, 28) and "l2.mlp.shared.up" not in s
    raw = cfg.to_json()
    assert raw["layers"][1]["mlp"] is None and raw["layers"][2]["mixer"]["kv_from"] == 1
    # the rank of the decay's projection may be left to the checkpoint
    del raw["layers"][0]["mixer"]["rank"]
    open_ = kx.KemiraxConfig.from_json(raw)
    assert open_.layers[0].mixer.rank is None and open_.tensor_shapes()["l0.mix.a1"] == (None, 36)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="recurrent"), "mixer type"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=-1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=16), "kv_from"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "experts"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=0), "experts"),
    (lambda c: c.update(architecture="Other"), "not a"),
])
def test_configurations_outside_the_design_are_refused(change, message):
    raw = _cfg().to_json()
    change(raw)
    with pytest.raises(ValueError, match=message):
        kx.KemiraxConfig.from_json(raw)


def test_registry_recognises_and_audits_checkpoints(tmp_path, capsys):
    import json

    from deepseek_v4_2080ti_b200.cli import inspect_safetensors
    from deepseek_v4_2080ti_b200.formats import safetensors_io
    from deepseek_v4_2080ti_b200.runtime import loader
    from pocketllm import EngineArgs
    from pocketllm.api.errors import ConfigurationError
    cfg = _cfg()
    kx.write_checkpoint(str(tmp_path), cfg, seed=1)
    raw, spec = loader.checkpoint_family(str(tmp_path))
    assert spec.name == "kemirax" and spec.dtypes == ("bfloat16", "float32") and "kemirax" in registry.checkpoint_families()
    state = {n: t.clone() for n, t in safetensors_io.read_checkpoint(str(tmp_path))}
    assert {n: tuple(t.shape) for n, t in state.items()} == cfg.tensor_shapes()
    for drop_rank in (False, True):
        if drop_rank:
            for i in (0, 3):
                del raw["layers"][i]["mixer"]["rank"]
            (tmp_path / "config.json").write_text(json.dumps(raw))
        assert inspect_safetensors.main([str(tmp_path), "--audit"]) == 0
        assert "audit ok=1" in capsys.readouterr().out
    assert spec.audit(raw, {**{n: tuple(t.shape) for n, t in state.items()}, "l0.mix.a1": (6, 35)})["wrong_shape"] == ["l0.mix.a1"]
    open_ = kx.KemiraxConfig.from_json(raw)
    assert kx.KemiraxWeights(open_, state, "cpu").layers[3].mix.m.rank == 32
    with pytest.raises(ValueError, match="decay projection"):
        kx.KemiraxWeights(open_, {**state, "l0.mix.a1": torch.zeros(7, 36)}, "cpu")
    with pytest.raises(ValueError, match="missing"):
        kx.KemiraxWeights(cfg, {n: t for n, t in state.items() if n != "l1.mix.dkv"}, "cpu")
    with pytest.raises(ValueError, match="shapes"):
        kx.KemiraxWeights(cfg, {**state, "l0.mlp.correction": torch.zeros(6)}, "cpu")
    with pytest.raises(ValueError, match="one rank"):
        spec.build(raw, str(tmp_path), "cpu", world=2)
    with pytest.raises(ConfigurationError, match="needs a GPU"):
        loader.load_runtime(EngineArgs(model=str(tmp_path), device="cpu"))


def test_build_subset_lists_existing_sources():
    from deepseek_v4_2080ti_b200 import build
    assert all((build.CSRC / "kernels" / s).exists() for s in kx.KERNEL_SOURCES)
    assert all((build.CSRC / "kernels" / s).exists() for s in build.PRECISE)


def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).double()


def test_plain_statement_of_the_recurrence():
    """The recurrence against its closed form, and a sequence continued from a kept state."""
    n, h, d, v = 9, 2, 3, 4
    q, k, vv = _rand(n, h, d, seed=1), _rand(n, h, d, seed=2), _rand(n, h, v, seed=3)
    la = -_rand(n, h, d, seed=4).abs()
    o, s = ref.gated_recurrence(q, k, vv, la)
    for t in range(n):
        want = torch.zeros(h, v).double()
        for u in range(t + 1):
            decay = torch.exp(la[u + 1:t + 1].sum(0))
            want = want + (q[t] * decay * k[u]).sum(-1, keepdim=True) * vv[u]
        assert torch.allclose(o[t], want)
    o1, s1 = ref.gated_recurrence(q[:4], k[:4], vv[:4], la[:4])
    o2, s2 = ref.gated_recurrence(q[4:], k[4:], vv[4:], la[4:], s1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(s2, s)


def test_plain_statement_of_the_rotation():
    rot = {"dims": 6, "base": 100.0}
    x = _rand(3, 2, 8, seed=5)
    y = ref.rotate_half(x, [0, 1, 50], rot)
    assert torch.allclose(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    a = 50 * 100.0 ** (-2 / 6)
    assert y[2, 1, 1].item() == pytest.approx(x[2, 1, 1].item() * math.cos(a) - x[2, 1, 4].item() * math.sin(a))
    assert y[2, 1, 4].item() == pytest.approx(x[2, 1, 4].item() * math.cos(a) + x[2, 1, 1].item() * math.sin(a))
    # slow dimensions are stretched by the factor, fast ones are not, and both tables of the package agree
    for rot in ({"dims": 16, "base": 10000.0, "scaling": {"factor": 8.0, "original": 256, "fast": 8.0, "slow": 1.0}},
                {"dims": 32, "base": 500.0, "scaling": YARN}, {"dims": 6, "base": 100.0, "scaling": None}):
        f, m = ref.yarn_frequencies(rot)
        g, mg = mixattn.yarn_freqs(rot["dims"], rot["base"], rot["scaling"], "cpu")
        assert torch.allclose(f, g, rtol=1e-12) and m == pytest.approx(mg)
    f, m = ref.yarn_frequencies({"dims": 16, "base": 10000.0, "scaling": {"factor": 8.0, "original": 256, "fast": 8.0, "slow": 1.0}})
    plain = 10000.0 ** (-torch.arange(0, 16, 2).double() / 16)
    assert f[0].item() == 1.0 and f[-1].item() == pytest.approx(plain[-1].item() / 8) and m == pytest.approx(1 + 0.1 * math.log(8))


def test_plain_statement_of_the_small_parts():
    h, amount = _rand(4, 3, seed=6), torch.tensor([0.0, 1.0, 0.25]).double()
    m = ref.token_shift(h, amount)
    assert torch.equal(m[:, 0], h[:, 0]) and torch.allclose(m[1:, 1], h[:-1, 1]) and m[0, 1] == 0
    assert m[0, 2].item() == pytest.approx(0.75 * h[0, 2].item()) and m[3, 2].item() == pytest.approx(0.75 * h[3, 2].item() + 0.25 * h[2, 2].item())
    z = torch.tensor([-800.0, -3.0, 0.0, 5.0, 800.0]).double()
    assert torch.allclose(ref.log_sigmoid(z), torch.nn.functional.logsigmoid(z)) and ref.log_sigmoid(z)[0] == -800
    # the correction moves the choice, not the weight; weights are not renormalised
    logits = torch.tensor([[2.0, 1.0, 0.0, -1.0]]).double()
    s = torch.softmax(logits, -1)[0]
    idx, w = ref.choose(logits, torch.tensor([0.0, 0.0, 0.0, 0.9]).double(), 2)
    assert sorted(idx[0].tolist()) == [0, 3] and sorted(w[0].tolist()) == pytest.approx(sorted([s[0].item(), s[3].item()]))
    # both factors of the unit are clamped, the first from above only
    eye = torch.eye(3).double()
    got = ref.clamped_unit(torch.tensor([[-50.0, 9.0, 0.5]]).double(), eye, eye, eye, 2.0)
    assert got[0].tolist() == pytest.approx([0.0, 2 / (1 + math.exp(-3.404)) * 3, 0.5 / (1 + math.exp(-0.851)) * 1.5])
    # an identity expert gives the input back, times its weight
    w = {"router": torch.zeros(2, 3).double(), "correction": torch.tensor([0.0, 1.0]).double(), "e0.gate": eye, "e0.up": eye, "e0.down": eye}
    mlp = {"expert": {"limit": 2.0}, "router": {"experts": 1, "identity": 1, "top": 1}}
    x = _rand(2, 3, seed=7)
    assert torch.allclose(ref.experts(x, w, mlp), 0.5 * x)


def test_plain_attention_sees_the_past_only_and_all_of_it():
    s = _rand(7, 7, seed=8)
    p = ref.causal_softmax(s)
    assert torch.allclose(p.sum(-1), torch.ones(7).double()) and not p.triu(1).any()
    assert torch.allclose(p[6], torch.softmax(s[6], -1)) and torch.allclose(p[:4, :4], ref.causal_softmax(s[:4, :4]))


def test_borrowed_keys_are_those_of_the_lending_layer():
    """Changing the lender's latent projection changes the borrower even where the lender adds nothing to the residual."""
    cfg = _cfg()
    state = dict(kx.synth_state(cfg, 3))
    state["l1.mix.o"] = torch.zeros_like(state["l1.mix.o"])
    toks = list(range(12))
    taps = []
    a = ref.forward(cfg.to_json(), state, toks, taps=taps)
    assert torch.equal(taps[1], taps[0])
    state["l1.mix.dkv"] = -state["l1.mix.dkv"]
    assert not torch.allclose(a, ref.forward(cfg.to_json(), state, toks))


def test_weight_layouts():
    """Padded and reordered weights give the statement's projections."""
    cfg = _cfg()
    state = {n: t.float() for n, t in kx.synth_state(cfg, 5)}
    w = kx.KemiraxWeights(cfg, state, "cpu", torch.float32)
    x = torch.zeros(4, w.ld)
    x[:, :36] = _rand(4, 36, seed=14).float()
    xs = x[:, :36]
    near = lambda a, b: torch.allclose(a, b, atol=1e-5)
    lw = w.layers[0]
    g = x @ lw.gates.w32.t()
    assert near(g[:, :36], xs @ state["l0.rg1"].t()) and near(g[:, w.ld:w.ld + 36], xs @ state["l0.rg2"].t()) and not g[:, 36:w.ld].any()
    assert torch.equal(lw.gate_b[:36], state["l0.rg1.b"]) and torch.equal(lw.gate_b[w.ld:w.ld + 36], state["l0.rg2.b"])
    assert lw.norm == pytest.approx(float(state["l0.norm1"])) and torch.equal(lw.shift[:36], state["l0.shift"])
    m = lw.mix.m
    p = x @ lw.mix.proj.w32.t()
    oq, ok, ov, og, oa = m.offsets
    assert (m.d, m.v, m.rank) == (16, 16, 16)
    for off, n, real, pad in ((oq, "q", 10, 16), (ok, "k", 10, 16), (ov, "v", 14, 16), (og, "g", 14, 16)):
        y = p[:, off:off + 3 * pad].view(4, 3, pad)
        assert near(y[..., :real], (xs @ state["l0.mix." + n].t()).view(4, 3, real)) and not y[..., real:].any()
    z = p[:, oa:oa + 16] @ m.w2.t() + m.b2
    assert near(z.view(4, 3, 16)[..., :10], ((xs @ state["l0.mix.a1"].t()) @ state["l0.mix.a2"].t() + state["l0.mix.a2.b"]).view(4, 3, 10))
    f = lw.ff
    r = x @ f.router.w32.t()
    assert near(r[:, :7], xs @ state["l0.mlp.router"].t()) and near(r[:, 7:8], xs @ state["l0.mlp.shared.sg"].t())
    w13 = f.w13.weight.view(5, 2, 32, w.ld)
    assert torch.equal(w13[3, 1, :22, :36], state["l0.mlp.e3.up"]) and not w13[:, :, 22:].any()
    assert torch.equal(f.w2.weight.view(5, w.ld, 32)[2, :36, :22], state["l0.mlp.e2.down"])
    t = decoder.GLU_TILE
    assert lw.gates.n == 256 and lw.wide.n >= 256 + f.up.n and torch.equal(lw.wide.w32[256:256 + f.up.n], f.up.w32)
    up = x @ f.up.w32.t()
    assert near(up[:, :30], xs @ state["l0.mlp.shared.gate"].t()) and near(up[:, t:t + 30], xs @ state["l0.mlp.shared.up"].t())
    # latent attention: both forms of the up projections
    a = w.layers[1].mix
    d = x @ a.down.w32.t()
    assert near(d[:, :20], xs @ state["l1.mix.dq"].t()) and near(d[:, 32:60], (xs @ state["l1.mix.dkv"].t())[:, :28])
    assert near(d[:, 64:70], (xs @ state["l1.mix.dkv"].t())[:, 28:]) and not d[:, 20:32].any() and not d[:, 60:64].any()
    q = torch.zeros(4, 32)
    q[:, :20] = _rand(4, 20, seed=15).float()
    qh = (q @ a.uq.w32.t())[:, :5 * 32].view(4, 5, 32)
    want = (q[:, :20] @ state["l1.mix.uq"].t()).view(4, 5, 18)
    assert near(qh[..., :12], want[..., :12]) and near(qh[..., 16:22], want[..., 12:]) and not qh[..., 12:16].any()
    c = torch.zeros(4, 32)
    c[:, :28] = _rand(4, 28, seed=16).float()
    keys = (c[:, :28] @ state["l1.mix.uk"].t()).view(4, 5, 12)
    lat = torch.einsum("thd,hcd->thc", qh[..., :16], a.uk)
    assert near((lat * c[:, None]).sum(-1), (want[..., :12] * keys).sum(-1))
    assert near(torch.einsum("tc,hvc->thv", c, a.uv)[..., :18], (c[:, :28] @ state["l1.mix.uv"].t()).view(4, 5, 18))
    assert a.ukv is None and w.layers[1].ff is None and w.layers[1].gates.n == w.ld and w.layers[2].mix.m.c_w is None
    bf = kx.KemiraxWeights(cfg, state, "cpu", torch.bfloat16).layers[1].mix
    both = bf.ukv.weight.view(5, 16 + 32, 32).float()
    assert torch.allclose(both[:, :12, :28].reshape(60, 28), state["l1.mix.uk"]) and torch.allclose(both[:, 16:34, :28].reshape(90, 28), state["l1.mix.uv"])


def test_contexts_of_a_mixed_step_are_laid_out_one_after_the_other():
    """``kv_start`` / ``kv_total`` of the tile entries: their whole contexts, in row order, single rows excluded."""
    from deepseek_v4_2080ti_b200.models.paged import PagedRuntime
    seen = []

    class Probe(PagedRuntime):
        tile_min_rows = 4

        def _next(self, logits):
            return logits.argmax(-1)

        def _forward(self, ids, positions, kv_slots, meta, rows):
            if meta["mode"] == "mixed" and meta["tile_rows"]:
                seen.append((meta["kv_start"].tolist(), meta["kv_len"].tolist(), meta["kv_total"], meta["q_start"].tolist()))
            return torch.zeros(rows.numel() if rows is not None else ids.numel(), 3)
    rt = Probe("cpu", max_slots=3, max_context=64, block_size=8)
    a, b, c = (rt.allocate() for _ in range(3))
    rt.step([(a, [1] * 5, []), (b, [1] * 2, []), (c, [1] * 9, [0])])
    rt.step([(b, [1] * 6, []), (a, [1], []), (c, [1] * 4, [0])])
    rt.step([(a, [1], [0]), (b, [1] * 2, [])])
    assert seen == [([0, 5], [5, 9], 14, [0, 5]), ([0, 8], [8, 13], 21, [0, 6])]
