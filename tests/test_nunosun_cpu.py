"""Nunosun decoder on the CPU: configuration and tensor inventory, registry, the plain statement's own invariants, and the weight
layouts of the serving path against it."""
import math

import pytest
import torch

from deepseek_v4_2080ti_b200.models import nunosun as ns, registry
from deepseek_v4_2080ti_b200.models.reference_cpu import nunosun_ref as ref
from deepseek_v4_2080ti_b200.ops import winattn


def _cfg():
    return ns.NunosunConfig(61, 36, 1e-4, 5, 3, 0.25, [
        ns.LayerSpec(ns.DeltaSpec(6, 3, 10, 14, 4), ns.DenseSpec(22)),
        ns.LayerSpec(ns.PairSpec(ns.WindowSpec(4, 2, 12, 18, 0.3, 7, 20, 8), ns.RetentionSpec(3, 10, 6, (0.5, 0.9, 1.0), 4, 500.0)), ns.ExpertsSpec(9, 3, 2)),
        ns.LayerSpec(ns.DeltaSpec(2, 2, 7, 9, 1)),
        ns.LayerSpec(ns.PairSpec(ns.WindowSpec(1, 1, 8, 8, 1.0, 1, 4, 5), ns.RetentionSpec(1, 8, 16, (0.25,), 8, 10.0)), ns.DenseSpec(40))])


def test_config_round_trip_and_inventory():
    cfg = _cfg()
    back = ns.NunosunConfig.from_json(cfg.to_json())
    for L in cfg.layers:                                       # the bias table's rows are the checkpoint's
        if isinstance(L.mixer, ns.PairSpec):
            L.mixer.left.buckets = None
    assert back == cfg and cfg.vocab_size == 61
    s = _cfg().tensor_shapes()
    assert s["side.embed"] == (61, 20) and s["embed.norm"] == s["final.norm"] == (36,)
    assert s["l0.canon1"] == (36, 3) and s["l0.side.gate"] == (5, 36) and s["l0.side.proj"] == (36, 5)
    assert s["l0.mix.q"] == (30, 36) and s["l0.mix.v"] == s["l0.mix.g"] == (84, 36) and s["l0.mix.v.conv"] == (84, 4) and s["l0.mix.a"] == (6, 36)
    assert s["l0.mlp.up"] == (22, 36) and s["l0.mlp.act"] == (4,) and s["l2.mix.k.conv"] == (14, 1) and not any(n.startswith("l2.mlp") for n in s)
    assert s["l1.mix.left.k"] == (24, 36) and s["l1.mix.left.v"] == (36, 36) and s["l1.mix.left.rel"] == (8, 4) and s["l1.mix.left.q.norm"] == (12,)
    assert s["l1.mix.right.v"] == (18, 36) and s["l1.mix.right.o"] == (36, 18) and s["l1.mix.right.out"] == (36,)
    assert s["l1.mlp.e2.down"] == (36, 9) and "l1.mlp.e3.up" not in s and s["l1.mlp.router.b"] == (3,)
    assert back.tensor_shapes()["l1.mix.left.rel"] == (None, 4)
    raw = cfg.to_json()
    assert raw["layers"][2]["mlp"] is None and raw["layers"][1]["mixer"]["left"]["mask"] == {"size": 7} and raw["logit_scale"] == 0.25


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="recurrent"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "convolution taps"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "window"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.9]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.9, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["right"]["rot"].update(dims=5), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["right"]["rot"].update(dims=12), "rot.dims"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "feed-forward kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=4), "experts"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=0), "experts"),
    (lambda c: c["canon"].update(taps=0), "canon.taps"),
    (lambda c: c.update(architecture="Other"), "not a"),
])
def test_configurations_outside_the_design_are_refused(change, message):
    raw = _cfg().to_json()
    change(raw)
    with pytest.raises(ValueError, match=message):
        ns.NunosunConfig.from_json(raw)


def test_registry_recognises_and_audits_checkpoints(tmp_path, capsys):
    from deepseek_v4_2080ti_b200.cli import inspect_safetensors
    from deepseek_v4_2080ti_b200.formats import safetensors_io
    from deepseek_v4_2080ti_b200.runtime import loader
    from pocketllm import EngineArgs
    from pocketllm.api.errors import ConfigurationError
    cfg = _cfg()
    ns.write_checkpoint(str(tmp_path), cfg, seed=1)
    raw, spec = loader.checkpoint_family(str(tmp_path))
    assert spec.name == "nunosun" and spec.dtypes == ("bfloat16", "float32") and "nunosun" in registry.checkpoint_families()
    state = {n: t.clone() for n, t in safetensors_io.read_checkpoint(str(tmp_path))}
    assert {n: tuple(t.shape) for n, t in state.items()} == cfg.tensor_shapes()
    assert inspect_safetensors.main([str(tmp_path), "--audit"]) == 0
    assert "audit ok=1" in capsys.readouterr().out
    assert spec.audit(raw, {**{n: tuple(t.shape) for n, t in state.items()}, "l1.mix.left.rel": (8, 3)})["wrong_shape"] == ["l1.mix.left.rel"]
    with pytest.raises(ValueError, match="missing"):
        ns.NunosunWeights(cfg, {n: t for n, t in state.items() if n != "l1.mix.right.out"}, "cpu")
    with pytest.raises(ValueError, match="shapes"):
        ns.NunosunWeights(cfg, {**state, "l0.mlp.act": torch.zeros(3)}, "cpu")
    open_ = ns.NunosunConfig.from_json(raw)
    with pytest.raises(ValueError, match="distance bias"):
        ns.NunosunWeights(open_, {**state, "l1.mix.left.rel": torch.zeros(40, 4)}, "cpu")
    with pytest.raises(ValueError, match="one rank"):
        spec.build(raw, str(tmp_path), "cpu", world=2)
    with pytest.raises(ConfigurationError, match="needs a GPU"):
        loader.load_runtime(EngineArgs(model=str(tmp_path), device="cpu"))


def test_build_subset_lists_existing_sources():
    from deepseek_v4_2080ti_b200 import build
    assert all((build.CSRC / "kernels" / s).exists() for s in ns.KERNEL_SOURCES)
    assert all((build.CSRC / "kernels" / s).exists() for s in build.PRECISE)


def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).double()


def test_plain_statement_of_the_recurrences():
    """Retention and the delta rule against their closed forms, and sequences continued from a kept state."""
    n, h, d, v = 9, 2, 3, 4
    q, k, vv = _rand(n, h, d, seed=1), _rand(n, h, d, seed=2), _rand(n, h, v, seed=3)
    decay = torch.tensor([0.5, 0.9]).double()
    o, s = ref.retention_recurrence(q, k, vv, decay)
    for t in range(n):
        want = sum((decay ** (t - u))[:, None] * (q[t] * k[u]).sum(-1, keepdim=True) * vv[u] for u in range(t + 1))
        assert torch.allclose(o[t], want)
    o1, s1 = ref.retention_recurrence(q[:4], k[:4], vv[:4], decay)
    o2, s2 = ref.retention_recurrence(q[4:], k[4:], vv[4:], decay, s1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(s2, s)
    # a unit key written with a full step reads back its value, whatever the state held in its direction
    ku, ld, beta = ref.unit(k), -_rand(n, h, seed=4).abs(), torch.sigmoid(_rand(n, h, seed=5))
    start = _rand(h, d, v, seed=6)
    one, _ = ref.delta_recurrence(ku[:1], ku[:1], vv[:1], ld[:1], torch.ones(1, h).double(), start)
    assert torch.allclose(one[0], vv[0], atol=1e-5)
    # the transition is (I - beta k k^T) times the decay
    o, s = ref.delta_recurrence(q, ku, vv, ld, beta, start)
    m = start.clone()
    for t in range(n):
        eye = torch.eye(d).double() - beta[t][:, None, None] * ku[t][:, :, None] * ku[t][:, None, :]
        m = eye @ (torch.exp(ld[t])[:, None, None] * m) + beta[t][:, None, None] * ku[t][:, :, None] * vv[t][:, None, :]
        assert torch.allclose(torch.einsum("hdv,hd->hv", m, q[t]), o[t])
    assert torch.allclose(m, s)
    o1, s1 = ref.delta_recurrence(q[:5], ku[:5], vv[:5], ld[:5], beta[:5], start)
    o2, s2 = ref.delta_recurrence(q[5:], ku[5:], vv[5:], ld[5:], beta[5:], s1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(s2, s)


def test_plain_statement_of_the_rotation():
    x = _rand(3, 2, 8, seed=5)
    y = ref.rotate_half(x, [0, 1, 50], 6, 100.0)
    assert torch.allclose(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    a = 50 * 100.0 ** (-2 / 6)
    assert y[2, 1, 1].item() == pytest.approx(x[2, 1, 1].item() * math.cos(a) - x[2, 1, 4].item() * math.sin(a))
    assert y[2, 1, 4].item() == pytest.approx(x[2, 1, 4].item() * math.cos(a) + x[2, 1, 1].item() * math.sin(a))


def test_plain_statement_of_the_small_parts():
    x, w = _rand(6, 2, seed=7), _rand(2, 3, seed=8)
    y = ref.causal_conv(x, w)
    assert torch.allclose(y[0], w[:, 2] * x[0]) and torch.allclose(y[4], w[:, 0] * x[2] + w[:, 1] * x[3] + w[:, 2] * x[4])
    assert torch.allclose(ref.causal_conv(x, w[:, 2:]), x * w[:, 2])
    z = torch.tensor([-800.0, -3.0, 0.0, 5.0, 800.0]).double()
    assert torch.allclose(ref.softplus(z), torch.nn.functional.softplus(z)) and ref.softplus(z)[-1] == 800
    assert torch.allclose(ref.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    c = torch.tensor([0.5, -2.0, 3.0, 0.25]).double()
    p = ref.poly_norm(torch.tensor([[1.0, -2.0]]).double(), c, 0.0)[0]
    r = [math.sqrt((1 + 4 ** i) / 2) for i in (1, 2, 3)]
    assert p.tolist() == pytest.approx([0.5 / r[0] - 2 / r[1] + 3 / r[2] + 0.25, -1.0 / r[0] - 8 / r[1] - 24 / r[2] + 0.25])
    # the weights are a softmax over the chosen logits only
    idx, wt = ref.choose(torch.tensor([[2.0, -5.0, 4.0, 3.0]]).double(), 2)
    assert idx[0].tolist() == [2, 3] and wt[0].tolist() == pytest.approx([1 / (1 + math.exp(-1)), 1 / (1 + math.exp(1))])


def test_distance_buckets():
    """One row per distance in the lower half, logarithmic steps above, the last row from the reach on; both tables agree."""
    b = [ref.bucket(n, 16, 64) for n in range(200)]
    assert b[:8] == list(range(8)) and b[8] == 8 and b[64:] == [15] * 136 and sorted(b) == b and set(b) == set(range(16))
    assert [n for n in range(1, 65) if b[n] != b[n - 1]][8:] == [11, 14, 18, 23, 30, 39, 50]      # 8 (64 / 8)^(i / 8), rounded up
    for rows, reach, size in ((16, 64, 200), (9, 40, 75), (4, 8, 1), (32, 1000, 3000), (14, 90, 37), (2, 3, 10)):
        assert winattn.distance_buckets(size, rows, reach).tolist() == [ref.bucket(n, rows, reach) for n in range(size)]
    rel = _rand(9, 3, seed=9).float()
    t = winattn.distance_bias(rel, 75, 40)
    assert t.shape == (3, 75) and torch.allclose(t[2, 50] * math.log(2.0), rel[ref.bucket(50, 9, 40), 2])


def test_plain_attention_sees_its_window_only():
    mix = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.5, "mask": {"size": 4}, "bias_max": 6}
    shapes = {"q": (8, 5), "k": (4, 5), "v": (3, 5), "q.norm": (4,), "k.norm": (4,), "rel": (4, 2), "o": (5, 6)}
    w = {n: _rand(*s, seed=20 + i) for i, (n, s) in enumerate(shapes.items())}
    h = _rand(12, 5, seed=30)
    y = ref.window_attention(h, w, mix, 1e-5)
    other = h.clone()
    other[3] += 1.0
    z = ref.window_attention(other, w, mix, 1e-5)
    moved = [not torch.allclose(a, b) for a, b in zip(y, z)]
    assert moved == [3 <= t <= 6 for t in range(12)]
    # the window is what a full softmax over those keys alone would give
    alone = ref.window_attention(h[5:9], w, mix, 1e-5)
    assert torch.allclose(alone[3], y[8])
    # the bias is not scaled: raising the row of one distance draws the weight there
    w["rel"][1] += 100.0
    v = h @ w["v"].t()
    assert torch.allclose(ref.window_attention(h, w, mix, 1e-5)[9], torch.cat([v[8], v[8]]) @ w["o"].t())


def test_every_part_of_a_layer_reaches_the_logits():
    cfg = _cfg()
    state = dict(ns.synth_state(cfg, 3))
    raw, toks = cfg.to_json(), list(range(14))
    base = ref.forward(raw, state, toks)
    for name, t in state.items():
        other = dict(state)
        # a common factor of normalised keys or of one decay's table would be no change of the function: perturb one element
        bump = torch.zeros_like(t.float())
        bump.view(-1)[bump.numel() // 3] = 0.5
        if name in ("embed", "side.embed"):
            bump[:14] = 0.5
        other[name] = t.float() + bump
        if name.endswith(("left.rel", "left.q.norm", "left.k.norm", "left.q", "left.k")) and name.startswith("l3."):
            continue                                             # a window of one key: scores do not matter
        if name.endswith("left.rel"):
            other[name] = t.float() * 2.0
        assert not torch.allclose(ref.forward(raw, other, toks), base, atol=1e-9), name


def test_weight_layouts():
    """Padded and reordered weights give the statement's projections."""
    cfg = _cfg()
    state = {n: t.float() for n, t in ns.synth_state(cfg, 5)}
    w = ns.NunosunWeights(cfg, state, "cpu", torch.float32)
    x = torch.zeros(4, w.ld)
    x[:, :36] = _rand(4, 36, seed=14).float()
    xs = x[:, :36]
    near = lambda a, b: torch.allclose(a, b, atol=1e-5)
    assert torch.equal(w.side_embed.view(61, 4, 16)[:, 2, :5], state["side.embed"][:, 10:15]) and not w.side_embed.view(61, 4, 16)[:, :, 5:].any()
    assert torch.allclose(w.final_norm[:36], 0.25 * state["final.norm"]) and not w.final_norm[36:].any()
    lw = w.layers[0]
    assert torch.allclose(lw.conv[:2, :36], state["l0.canon1"][:, :2].t()) and torch.allclose(lw.conv[2, :36], 1 + state["l0.canon1"][:, 2])
    m = lw.mix.m
    p = x @ lw.mix.proj.w32.t()
    at = 0
    for n, h, real, pad in (("q", 3, 10, 16), ("k", 3, 10, 16), ("v", 6, 14, 16), ("g", 6, 14, 16)):
        y = p[:, at:at + h * pad].view(4, h, pad)
        assert near(y[..., :real], (xs @ state["l0.mix." + n].t()).view(4, h, real)) and not y[..., real:].any()
        if n != "g":
            c = m.conv[:, at:at + h * pad].view(4, h, pad)
            assert torch.equal(c[..., :real], state[f"l0.mix.{n}.conv"].t().reshape(4, h, real)) and not c[..., real:].any()
        at += h * pad
    assert near(p[:, at:at + 6], xs @ state["l0.mix.a"].t()) and near(p[:, at + 6:at + 12], xs @ state["l0.mix.b"].t()) and m.channels == 192
    assert torch.allclose(m.neg_a, -torch.exp(state["l0.mix.A_log"]))
    assert lw.ff.up.n == lw.ff.down.k == 32 and torch.equal(lw.ff.down.w32[:36, :22], state["l0.mlp.down"]) and len(lw.ff.act) == 4
    pw = w.layers[1].mix
    p, at = x @ pw.proj.w32.t(), 0
    for n, h, real, pad in (("left.q", 4, 12, 16), ("left.k", 2, 12, 16), ("left.v", 2, 18, 32), ("right.q", 3, 10, 16), ("right.k", 3, 10, 16),
                            ("right.v", 3, 6, 16), ("right.g", 3, 6, 16)):
        if n == "right.q":
            assert at == pw.right_off
        y = p[:, at:at + h * pad].view(4, h, pad)
        assert near(y[..., :real], (xs @ state["l1.mix." + n].t()).view(4, h, real)) and not y[..., real:].any()
        at += h * pad
    assert torch.allclose(pw.left_w[:36], 0.5 * state["l1.mix.left.out"]) and torch.allclose(pw.right_w[:36], 0.5 * state["l1.mix.right.out"])
    z = torch.zeros(4, 4, 32)
    z[..., :18] = _rand(4, 4, 18, seed=15).float()
    assert near((z.view(4, -1) @ pw.left_o.w32.t())[:, :36], z[..., :18].reshape(4, -1) @ state["l1.mix.left.o"].t())
    assert pw.right.decay.tolist() == pytest.approx([0.5, 0.9, 1.0]) and pw.right.log2_decay.tolist() == pytest.approx([-1.0, math.log2(0.9), 0.0])
    f = w.layers[1].ff
    w13 = f.w13.weight.view(3, 2, 16, w.ld)
    assert torch.equal(w13[2, 1, :9, :36], state["l1.mlp.e2.up"]) and not w13[:, :, 9:].any()
    assert torch.equal(f.w2.weight.view(3, w.ld, 16)[1, :36, :9], state["l1.mlp.e1.down"]) and torch.equal(f.router_b, state["l1.mlp.router.b"])
    assert w.layers[2].ff is None and w.nbytes() > 0


def test_pages_in_front_of_the_longest_window_go_back():
    class Shell(ns.NunosunRuntime):
        def __init__(self, window):
            self.window = window
    for window, length, floor in ((7, 3, 0), (7, 6, 0), (7, 7, 1), (7, 50, 44), (1, 9, 9), (0, 9, 9)):
        rt = Shell(window)
        assert rt.history_floor(length) == floor and rt.history_span() == max(window - 1, 0)
        assert length - rt.history_floor(length) <= rt.history_span() or length < window
