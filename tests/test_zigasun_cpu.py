"""Zigasun decoder on the CPU: configuration and tensor inventory, registry, the plain statement's own invariants, and the
weight layouts of the serving path against it."""
import math

import pytest
import torch

from deepseek_v4_2080ti_b200.models import registry, zigasun as zg
from deepseek_v4_2080ti_b200.models.reference_cpu import zigasun_ref as ref
from deepseek_v4_2080ti_b200.ops import decoder, scan


def _cfg():
    return zg.ZigasunConfig(61, 36, 1e-4, 2.5, 0.6, [
        zg.LayerSpec(zg.ScanSpec(50, 5, 3, 3), 22, 1.5),
        zg.LayerSpec(zg.AttentionSpec(6, 2, 10, 14, 0.3, 0.2, 0.4, 9.0), 0, 0.0),
        zg.LayerSpec(zg.AttentionSpec(4, 2, 10, 14, 0.2, 0.5, kv_from=1), 30, 0.7),
        zg.LayerSpec(zg.ScanSpec(24, 9, 20, 1))])


def test_config_round_trip_and_inventory():
    cfg = _cfg()
    assert zg.ZigasunConfig.from_json(cfg.to_json()) == cfg and cfg.vocab_size == 61
    s = cfg.tensor_shapes()
    assert s["l0.mix.in"] == (100, 36) and s["l0.mix.x"] == (13, 50) and s["l0.mix.conv"] == (50, 3) and s["l0.mlp.down"] == (36, 22)
    assert s["l1.mix.q"] == (120, 36) and s["l1.mix.v"] == (28, 36) and s["l1.mix.o"] == (36, 84) and s["l1.mix.g"] == (6, 36)
    assert "l1.norm2" not in s and "l2.mix.k" not in s and "l2.mix.v" not in s and "l2.mix.k.norm" not in s
    assert s["l2.mix.q"] == (80, 36) and s["l2.norm2"] == (36,) and "l3.mlp.up" not in s
    raw = cfg.to_json()
    assert "q_temp" not in raw["layers"][2]["mixer"] and raw["layers"][2]["mixer"]["kv_from"] == 1


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="recurrent"), "mixer type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=-1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "kv_from"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda c: c.update(architecture="Other"), "not a"),
])
def test_configurations_outside_the_design_are_refused(change, message):
    raw = _cfg().to_json()
    change(raw)
    with pytest.raises(ValueError, match=message):
        zg.ZigasunConfig.from_json(raw)


def test_registry_recognises_and_audits_checkpoints(tmp_path, capsys):
    from deepseek_v4_2080ti_b200.cli import inspect_safetensors
    from deepseek_v4_2080ti_b200.formats import safetensors_io
    from deepseek_v4_2080ti_b200.runtime import loader
    from pocketllm import EngineArgs
    from pocketllm.api.errors import ConfigurationError
    cfg = _cfg()
    zg.write_checkpoint(str(tmp_path), cfg, seed=1)
    raw, spec = loader.checkpoint_family(str(tmp_path))
    assert spec.name == "zigasun" and spec.dtypes == ("bfloat16", "float32") and "zigasun" in registry.checkpoint_families()
    state = {n: t.clone() for n, t in safetensors_io.read_checkpoint(str(tmp_path))}
    assert {n: tuple(t.shape) for n, t in state.items()} == cfg.tensor_shapes()
    assert inspect_safetensors.main([str(tmp_path), "--audit"]) == 0
    assert "audit ok=1" in capsys.readouterr().out
    with pytest.raises(ValueError, match="missing"):
        zg.ZigasunWeights(cfg, {n: t for n, t in state.items() if n != "l1.mix.g"}, "cpu")
    with pytest.raises(ValueError, match="shapes"):
        zg.ZigasunWeights(cfg, {**state, "l0.mix.D": torch.zeros(49)}, "cpu")
    with pytest.raises(ValueError, match="one rank"):
        spec.build(raw, str(tmp_path), "cpu", world=2)
    with pytest.raises(ConfigurationError, match="needs a GPU"):
        loader.load_runtime(EngineArgs(model=str(tmp_path), device="cpu"))


def test_build_subset_lists_existing_sources():
    from deepseek_v4_2080ti_b200 import build
    assert all((build.CSRC / "kernels" / s).exists() for s in zg.KERNEL_SOURCES)
    assert all((build.CSRC / "kernels" / s).exists() for s in build.PRECISE)


def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).double()


def test_plain_statement_of_the_scan():
    """The recurrence against its closed form, and a sequence continued from a kept state."""
    n, c, st = 9, 3, 2
    x, b, cc, d = _rand(n, c, seed=1), _rand(n, st, seed=2), _rand(n, st, seed=3), _rand(c, seed=4)
    dt, a = _rand(n, c, seed=5).abs(), -_rand(c, st, seed=6).abs()
    y, s = ref.selective_scan(x, dt, a, b, cc, d)
    for t in range(n):
        want = d * x[t]
        for u in range(t + 1):
            decay = torch.exp(a * dt[u + 1:t + 1].sum(0)[:, None])
            want = want + (decay * (dt[u] * x[u])[:, None] * b[u] * cc[t]).sum(-1)
        assert torch.allclose(y[t], want)
    y1, s1 = ref.selective_scan(x[:4], dt[:4], a, b[:4], cc[:4], d)
    y2, s2 = ref.selective_scan(x[4:], dt[4:], a, b[4:], cc[4:], d, s1)
    assert torch.allclose(torch.cat([y1, y2]), y) and torch.allclose(s2, s)


def test_plain_statement_of_the_small_parts():
    x, w = _rand(6, 2, seed=7), _rand(2, 3, seed=8)
    y = ref.causal_conv(x, w, torch.tensor([0.5, -1.0]).double())
    assert torch.allclose(y[0], torch.tensor([0.5, -1.0]).double() + w[:, 2] * x[0])
    assert torch.allclose(y[4, 1], -1.0 + w[1, 2] * x[4, 1] + w[1, 1] * x[3, 1] + w[1, 0] * x[2, 1])
    z = torch.tensor([-800.0, -3.0, 0.0, 5.0, 800.0]).double()
    assert torch.allclose(ref.softplus(z), torch.nn.functional.softplus(z)) and ref.softplus(z)[4] == 800
    f = ref.query_temperature([0, 6, 7, 13, 14, 99], 0.5, 7)
    # the factor changes on the last position of a block
    assert f.tolist() == pytest.approx([1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3),
                                        1 + 0.5 * math.log(3), 1 + 0.5 * math.log(15)])
    lq = {n: torch.tensor(v).double() for n, v in (("lq1", [1.0, 2.0]), ("lk1", [0.5, 0.25]), ("lq2", [1.0, -1.0]), ("lk2", [0.0, 0.0]))}
    assert float(ref.lambda_of(lq, 0.3)) == pytest.approx(math.e - 1 + 0.3)
    a1, a2 = _rand(5, seed=9), _rand(5, seed=10)
    o = ref.difference_of_maps(a1, a2, torch.tensor(0.4).double(), 0.3, 0.0)
    assert float((o * o).mean()) == pytest.approx(0.49) and torch.allclose(o / o.norm(), (a1 - 0.4 * a2) / (a1 - 0.4 * a2).norm())
    # both factors of the gated unit are clamped, the first from above only
    eye = torch.eye(3).double()
    h = torch.tensor([[-50.0, 9.0, 0.5]]).double()
    got = ref.clamped_glu(h, {"gate": eye, "up": eye, "down": eye}, 2.0)
    assert got[0].tolist() == pytest.approx([0.0, 2 / (1 + math.exp(-3.404)) * 3, 0.5 / (1 + math.exp(-0.851)) * 1.5])


def test_plain_attention_sees_the_past_only():
    q, k, v = _rand(7, 4, seed=11), _rand(7, 4, seed=12), _rand(7, 3, seed=13)
    full = ref.softmax_attention(q, k, v, 0.7)
    for n in (1, 4):
        assert torch.allclose(full[:n], ref.softmax_attention(q[:n], k[:n], v[:n], 0.7))
    p = torch.exp(q[6] @ k.t() * 0.7)
    assert torch.allclose(full[6], p @ v / p.sum())


def test_borrowed_keys_are_those_of_the_lending_layer():
    """Changing the lender's key projection changes the borrower; the borrower's output without the lender's tensors cannot be
    formed from its own input."""
    cfg = _cfg()
    state = dict(zg.synth_state(cfg, 3))
    toks = list(range(12))
    a = ref.forward(cfg.to_json(), state, toks)
    taps, taps2 = [], []
    ref.forward(cfg.to_json(), state, toks, taps=taps)
    state2 = dict(state)
    state2["l1.mix.k"] = -state["l1.mix.k"]
    state2["l1.norm1"] = torch.zeros_like(state["l1.norm1"])
    state["l1.norm1"] = torch.zeros_like(state["l1.norm1"])      # layer 1 adds nothing: only its keys and values matter
    b = ref.forward(cfg.to_json(), state, toks, taps=taps2)
    assert torch.equal(taps2[1], taps2[0]) and not torch.allclose(a, b)
    assert not torch.allclose(b, ref.forward(cfg.to_json(), state2, toks))


def test_weight_layouts():
    """Padded and reordered weights give the statement's projections: interleaved gate / up tiles, padded heads, the parts of
    the scan's projections, and the step-size projection that reads the whole row."""
    cfg = _cfg()
    state = {n: t.float() for n, t in zg.synth_state(cfg, 5)}
    w = zg.ZigasunWeights(cfg, state, "cpu", torch.float32)
    x = torch.zeros(4, w.ld)
    x[:, :36] = _rand(4, 36, seed=14).float()
    xs = x[:, :36]
    lw = w.layers[0]
    t = decoder.GLU_TILE
    z = x @ lw.up.w32.t()
    assert lw.up.n % (2 * t) == 0 and torch.allclose(z[:, :22], xs @ state["l0.mlp.gate"].t(), atol=1e-5)
    assert torch.allclose(z[:, t:t + 22], xs @ state["l0.mlp.up"].t(), atol=1e-5) and not z[:, 22:t].any() and not z[:, t + 22:].any()
    assert torch.equal(lw.down.w32[:36, :22], state["l0.mlp.down"]) and not lw.down.w32[:, 22:].any()
    assert torch.allclose(lw.norm1[:36], 0.6 * state["l0.norm1"])
    s = lw.mix
    xz = x @ s.in_.w32.t()
    assert s.inner == 64 and torch.allclose(xz[:, :50], xs @ state["l0.mix.in"][:50].t(), atol=1e-5)
    assert torch.allclose(xz[:, 64:114], xs @ state["l0.mix.in"][50:].t(), atol=1e-5) and not xz[:, 50:64].any()
    h = torch.zeros(4, 64)
    h[:, :50] = _rand(4, 50, seed=15).float()
    p = h @ s.x.w32.t()
    want = h[:, :50] @ state["l0.mix.x"].t()
    assert (s.b_off, s.c_off) == (8, 16) and torch.allclose(p[:, :3], want[:, :3], atol=1e-5)
    assert torch.allclose(p[:, 8:13], want[:, 3:8], atol=1e-5) and torch.allclose(p[:, 16:21], want[:, 8:], atol=1e-5)
    assert torch.allclose((p @ s.dt.w32.t())[:, :50], want[:, :3] @ state["l0.mix.dt"].t(), atol=1e-4)
    assert torch.allclose(s.a[:50], -torch.exp(state["l0.mix.A_log"])) and torch.equal(s.conv[:, :50], state["l0.mix.conv"].t())
    a = w.layers[1].mix
    y = x @ a.proj.w32.t()
    q = y[:, :a.m.q_width].view(4, 6, 2, 16)
    assert torch.allclose(q[..., :10], (xs @ state["l1.mix.q"].t()).view(4, 6, 2, 10), atol=1e-5) and not q[..., 10:].any()
    v = y[:, a.m.q_width + a.m.k_width:a.gate_off].view(4, 2, 16)
    assert torch.allclose(v[..., :14], (xs @ state["l1.mix.v"].t()).view(4, 2, 14), atol=1e-5)
    assert torch.allclose(y[:, a.gate_off:a.gate_off + 6], xs @ state["l1.mix.g"].t(), atol=1e-5)
    b = w.layers[2].mix
    assert b.m.k_w is None and b.gate_off == b.m.q_width and b.m.temp_every == 0.0
    assert b.m.lam == pytest.approx(float(ref.lambda_of({n: state["l2.mix." + n] for n in ("lq1", "lk1", "lq2", "lk2")}, 0.5)), abs=1e-5)
    bf = zg.ZigasunWeights(cfg, state, "cpu", torch.bfloat16).layers[0].mix.a
    assert torch.allclose(torch.exp2(0.3 * bf[:50]), torch.exp(-0.3 * torch.exp(state["l0.mix.A_log"])), rtol=1e-6)


def test_rows_are_padded_to_whole_tiles_only_where_it_is_cheap():
    make = lambda n: decoder.Projection.make(torch.ones(n, 32), torch.float32, "cpu", tile_n=True).n
    assert [make(n) for n in (5, 250, 256, 260, 300, 3088, 2304)] == [16, 256, 256, 272, 304, 3328, 2304]


def test_segments_describe_mixed_and_decode_batches():
    """A stand-in model with a running state per slot: it only sees the segments, and must reproduce each request alone."""
    import random

    from deepseek_v4_2080ti_b200.models.paged import PagedRuntime

    class Running(PagedRuntime):
        tile_min_rows = 4

        def __init__(self, **kw):
            super().__init__("cpu", **kw)
            self.state = self.slot_state(1, dtype=torch.int64, name="running sum")
            self.state.fill_(999)                                # an earlier request's leftovers

        def _next(self, logits):
            return logits.argmax(-1).to(torch.int32)

        def _forward(self, ids, positions, kv_slots, meta, rows):
            seg = meta["segments"]
            assert isinstance(seg, scan.Segments)
            assert seg.max_length == int(seg.length.max()) and seg.min_length <= int(seg.length.min())
            out, seen = torch.zeros(ids.numel(), 101), 0
            for f, n, slot in zip(seg.first.tolist(), seg.length.tolist(), seg.slot.tolist()):
                s = 7 if int(positions[f]) == 0 else int(self.state[slot])
                for r in range(f, f + n):
                    assert int(seg.row_first[r]) == f and int(seg.row_slot[r]) == slot
                    s = (s * 31 + int(ids[r]) + int(positions[r])) % 101
                    out[r, s] = 1
                    seen += 1
                self.state[slot] = s
            assert seen == ids.numel()
            return out if rows is None else out[rows.long()] if rows.numel() else None

    def alone(toks):
        s, res = 7, []
        for p, t in enumerate(toks):
            s = (s * 31 + t + p) % 101
            res.append(s)
        return res
    rng = random.Random(4)
    rt = Running(max_slots=3, max_context=64, block_size=8)
    assert rt.state.shape == (4, 1) and rt.scratch_slot == 3
    live = {}
    for _ in range(200):
        while len(live) < 3 and rng.random() < 0.6:
            live[rt.allocate()] = []
        entries, want = [], []
        for slot, hist in live.items():
            n = min(rng.choice([0, 1, 1, 2, 3, 4, 9]), 60 - len(hist))
            if n <= 0:
                continue
            hist += [rng.randrange(97) for _ in range(n)]
            places = sorted(rng.sample(range(n), rng.randint(1, n)))
            entries.append((slot, hist[-n:], places))
            want += [alone(hist)[len(hist) - n + w] for w in places]
        if entries:
            assert rt.step(entries).argmax(-1).tolist() == want
        for slot in [s for s, h in live.items() if len(h) >= 55 or rng.random() < 0.05]:
            rt.free(slot)
            live.pop(slot)
