"""Rutulix decoder on the CPU: configuration and tensor inventory, registry, the plain statement's own invariants, and the
host-side tables of the serving path against it."""
import math

import pytest
import torch

from deepseek_v4_2080ti_b200.models import registry, rutulix as rx
from deepseek_v4_2080ti_b200.models.reference_cpu import rutulix_ref as ref
from deepseek_v4_2080ti_b200.ops import mixattn


def _cfg():
    a = rx.AttentionSpec(6, 2, 20, 0.2, 7, 12, 700.0, {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0})
    b = rx.AttentionSpec(3, 3, 10, 0.4, 0, 10, 90.0, None)
    return rx.RutulixConfig(53, 36, 1e-4, [rx.LayerSpec(a, 44), rx.LayerSpec(b, 0), rx.LayerSpec(a, 18)], (1, 3, 3))


def test_config_round_trip_runs_and_inventory():
    cfg = _cfg()
    assert rx.RutulixConfig.from_json(cfg.to_json()) == cfg and cfg.vocab_size == 53
    assert cfg.runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None)]
    assert cfg.runs() == ref.layer_runs(3, cfg.to_json()["loop"])
    shapes = cfg.tensor_shapes()
    assert shapes["loop.step"] == (3, 36) and shapes["l0.mix.k"] == (40, 36) and shapes["l1.mix.talk"] == (3, 3)
    assert "l1.norm2" not in shapes and "l1.mlp.up" not in shapes and shapes["l2.mlp.down"] == (36, 18)
    cfg.loop = None
    assert "loop.step" not in cfg.tensor_shapes() and cfg.runs() == [(0, None), (1, None), (2, None)]
    assert rx.RutulixConfig.from_json(cfg.to_json()) == cfg


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="recurrent"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "rot.dims"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "feed-forward kind"),
    (lambda c: c.update(loop={"start": 1, "stop": 9, "times": 2}), "loop"),
    (lambda c: c.update(architecture="Other"), "not a"),
])
def test_configurations_outside_the_design_are_refused(change, message):
    raw = _cfg().to_json()
    change(raw)
    with pytest.raises(ValueError, match=message):
        rx.RutulixConfig.from_json(raw)


def test_registry_recognises_and_audits_checkpoints(tmp_path, capsys):
    from deepseek_v4_2080ti_b200.cli import inspect_safetensors
    from deepseek_v4_2080ti_b200.formats import safetensors_io
    from deepseek_v4_2080ti_b200.runtime.loader import checkpoint_family
    cfg = _cfg()
    rx.write_checkpoint(str(tmp_path), cfg, seed=1)
    raw, spec = checkpoint_family(str(tmp_path))
    assert spec.name == "rutulix" and spec.dtypes == ("bfloat16", "float32") and "rutulix" in registry.checkpoint_families()
    assert registry.detect_checkpoint({"architectures": ["Qwen3_5ForConditionalGeneration"]}) is None
    assert checkpoint_family(str(tmp_path / "nothing")) == (None, None)
    state = {n: t.clone() for n, t in safetensors_io.read_checkpoint(str(tmp_path))}
    assert {n: tuple(t.shape) for n, t in state.items()} == cfg.tensor_shapes()
    assert inspect_safetensors.main([str(tmp_path), "--audit"]) == 0
    assert "audit ok=1" in capsys.readouterr().out
    rep = spec.audit(raw, {**{n: tuple(t.shape) for n, t in state.items() if n != "head"}, "extra": (1,), "embed": (1, 1)})
    assert (rep["missing"], rep["unexpected"], rep["wrong_shape"], rep["ok"]) == (["head"], ["extra"], ["embed"], False)
    with pytest.raises(ValueError, match="missing"):
        rx.RutulixWeights(cfg, {n: t for n, t in state.items() if n != "head"}, "cpu")
    with pytest.raises(ValueError, match="one rank"):
        spec.build(raw, str(tmp_path), "cpu", world=2)
    with pytest.raises(ValueError, match="dtype"):
        spec.build(raw, str(tmp_path), "cpu", dtype="float16")


def test_no_host_path_for_the_family(tmp_path):
    from deepseek_v4_2080ti_b200.runtime import loader
    from pocketllm import EngineArgs
    from pocketllm.api.errors import ConfigurationError
    rx.write_checkpoint(str(tmp_path), _cfg())
    with pytest.raises(ConfigurationError, match="needs a GPU"):
        loader.load_runtime(EngineArgs(model=str(tmp_path), device="cpu"))


def test_trace_runner_refuses_what_it_cannot_run(tmp_path, capsys):
    from deepseek_v4_2080ti_b200.cli.trace_run import main
    assert main(["--model", str(tmp_path), "--out", str(tmp_path), "--max-tokens", "64"]) == 2
    (tmp_path / "config.json").write_text('{"dim": 8, "n_layers": 1, "n_routed_experts": 2, "kv_lora_rank": 4, "q_lora_rank": 4}')
    from deepseek_v4_2080ti_b200.runtime.loader import checkpoint_family
    if checkpoint_family(str(tmp_path))[1] is not None:
        assert main(["--model", str(tmp_path), "--out", str(tmp_path), "--max-tokens", "64", "--dtype", "float32"]) == 3


@pytest.mark.parametrize("dims,base,scaling", [
    (8, 10000.0, None), (16, 500.0, {"factor": 4.0, "original": 128, "fast": 16.0, "slow": 1.0}),
    (64, 2e5, {"factor": 1.0, "original": 4096, "fast": 32.0, "slow": 2.0}),
    (2, 50.0, {"factor": 8.0, "original": 32, "fast": 4.0, "slow": 4.0}),
    (40, 3000.0, {"factor": 2.5, "original": 100000, "fast": 64.0, "slow": 0.5})])
def test_frequency_tables(dims, base, scaling):
    f, m = mixattn.yarn_freqs(dims, base, scaling, "cpu")
    want, wm = ref.yarn_frequencies(dims, base, scaling)
    assert f.dtype == torch.float64 and f.numel() == dims // 2
    assert max(abs(a - b) for a, b in zip(f.tolist(), want)) < 1e-14 and abs(m - wm) < 1e-14
    if scaling:
        assert m == pytest.approx(0.1 * math.log(scaling["factor"]) + 1.0)
        plain = ref.yarn_frequencies(dims, base, None)[0]
        assert all(p / scaling["factor"] - 1e-12 <= x <= p + 1e-12 for p, x in zip(plain, want))


def test_rotation_is_relative_and_leaves_the_tail():
    gen = torch.Generator().manual_seed(0)
    q, k = torch.randn(1, 1, 12, generator=gen).double(), torch.randn(1, 1, 12, generator=gen).double()
    freqs, ms = ref.yarn_frequencies(8, 100.0, {"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0})
    rot = lambda x, p: ref.rotate_interleaved(x, torch.tensor([p]), freqs, ms)
    dot = lambda a, b: float((rot(q, a) * rot(k, b))[..., :8].sum())
    assert dot(9, 4) == pytest.approx(dot(105, 100)) and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    assert torch.equal(rot(q, 9)[..., 8:], q[..., 8:])


def test_plain_statement_mechanisms():
    gen = torch.Generator().manual_seed(3)
    x = torch.randn(5, 9, generator=gen).double() * 3 + 2
    y = ref.layer_norm(x, torch.ones(9).double(), 0.0)
    assert y.mean(-1).abs().max() < 1e-12 and (y.pow(2).mean(-1) - 1).abs().max() < 1e-12
    vis = ref.chunk_visible(10, 4)
    assert vis[7].nonzero().flatten().tolist() == [4, 5, 6, 7] and vis[8].nonzero().flatten().tolist() == [8]
    act = torch.tensor([0.3, -0.7]).double()
    z = torch.tensor([-40.0, -1e-4, 0.0, 1e-4, 5.0]).double()
    got = ref.xielu(z, act)
    ap, an = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.7))
    assert got[4] == pytest.approx(ap * 25 + 2.5) and got[0] == pytest.approx(an * 39 - 20) and got[2] == 0
    # an identity mixing matrix is ordinary grouped attention; a permutation swaps the heads' scores, not their values
    q, k, v = (torch.randn(6, h, 4, generator=gen).double() for h in (4, 2, 2))
    eye = torch.eye(4).double()
    plain = ref.talking_attention(q, k, v, eye, 0.5, ref.chunk_visible(6, None))
    s = (q[:, 3] @ k[:, 1].t() * 0.5).masked_fill(~ref.chunk_visible(6, None), float("-inf")).softmax(-1)
    assert torch.allclose(plain[:, 3], s @ v[:, 1])
    swapped = ref.talking_attention(q, k, v, eye[[3, 1, 2, 0]], 0.5, ref.chunk_visible(6, None))
    assert torch.allclose(swapped[:, 0], s @ v[:, 0])


def test_folding_the_mixing_into_the_queries_is_exact():
    """sum_g T[h, g] (q_g . k_kv(g)) equals one dot product with all key heads side by side."""
    gen = torch.Generator().manual_seed(5)
    H, G, D = 6, 3, 5
    q, k, talk = torch.randn(H, D, generator=gen).double(), torch.randn(G, D, generator=gen).double(), torch.randn(H, H, generator=gen).double()
    folded = torch.einsum("hcr,crd->hcd", talk.view(H, G, H // G), q.view(G, H // G, D)).reshape(H, G * D)
    raw = torch.stack([q[g] @ k[g // (H // G)] for g in range(H)])
    assert torch.allclose(folded @ k.reshape(-1), talk @ raw)


def test_history_bounds():
    class Shell(rx.RutulixRuntime):
        def __init__(self, chunks):
            self.chunks, self.block_size = chunks, 16
    rt = Shell([12, 30])
    assert [rt.history_floor(p) for p in (0, 11, 12, 29, 30, 35, 36, 60)] == [0, 0, 0, 0, 24, 24, 30, 60]
    assert rt.history_span() == 29 and rt.pages_held(1000, 8) == 4 and rt.pages_held(20, 8) == 2
    assert Shell([12, 0]).history_span() is None and Shell([12, 0]).history_floor(500) == 0
    for s in range(200):
        assert s - rt.history_floor(s) <= rt.history_span()


def test_build_subset_lists_existing_sources():
    from deepseek_v4_2080ti_b200 import build
    assert all((build.CSRC / "kernels" / s).exists() for s in rx.KERNEL_SOURCES)
    assert all((build.CSRC / "kernels" / s).exists() for s in build.PRECISE)
