"""Nunosun decoder: layers whose mixer and feed-forward read one norm side by side; what the mixer reads goes through a short
causal convolution first, and every layer adds a gated part of the token's side embedding.  Mixers are the gated delta rule and
a pair on the same rows: attention with a sliding window and a learned distance bias beside retention, each normalised before
the two are averaged.  Feed-forwards are dense with a polynomial of row norms, or routed experts.

The layers are described by config.json (sizes, order, constants); the passes, the pages, the state slots and the batching
come from ``models/paged.py``, the kernels from ``ops/winattn.py``, ``ops/decay.py``, ``ops/moe.py`` and ``ops/decoder.py``.
Activations are bf16 (serving) or fp32 (``dtype``).
"""
from __future__ import annotations

import contextlib
import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Iterator

import torch

from ..ops import decay, decoder, gemm, moe, winattn
from ..ops.decay import DeltaRule, Retention
from ..ops.decoder import Projection, Routed, cat_rows, pad16, pad_heads
from ..ops.winattn import WindowAttention
from ..utils import canary
from .paged import PagedRuntime

ARCH = "Nunosun"
# kernel sources the runtime launches (a partial build compiles only these)
KERNEL_SOURCES = ("branch_step.cu", "row_act.cu", "conv_rows.cu", "qk_head_prep.cu", "attn_window_rows.cu", "attn_window_prefill.cu", "decay_rule.cu",
                  "retention_chunk.cu", "delta_chunk.cu", "gated_linear.cu", "head_linear.cu", "moe.cu", "bias_act.cu", "gemm_f32.cu", "gemm_wdec.cu", "gemm_bf16_2cta.cu",
                  "elementwise.cu", "sampling.cu", "bounds.cu")


# ---------------------------------------------------------------------------------------------- configuration
@dataclass
class WindowSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    size: int
    reach: int                        # distances from here on share the last row of the bias table
    buckets: int | None = None        # rows of the bias table; None: what the checkpoint's tensor has


@dataclass
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot_dims: int
    rot_base: float


@dataclass
class PairSpec:
    left: WindowSpec
    right: RetentionSpec


@dataclass
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                         # taps


@dataclass
class DenseSpec:
    ff: int


@dataclass
class ExpertsSpec:
    ff: int
    experts: int
    top: int


@dataclass
class LayerSpec:
    mixer: PairSpec | DeltaSpec
    mlp: DenseSpec | ExpertsSpec | None = None


@dataclass
class NunosunConfig:
    vocab: int
    width: int
    eps: float
    side: int                         # values of the side embedding per layer
    taps: int                         # of the convolution in front of the mixers
    logit_scale: float = 1.0
    layers: list[LayerSpec] = field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def is_nunosun_json(raw: Any) -> bool:
        return isinstance(raw, dict) and raw.get("architecture") == ARCH

    @staticmethod
    def from_json(raw: dict) -> "NunosunConfig":
        if not NunosunConfig.is_nunosun_json(raw):
            raise ValueError(f"not a {ARCH} configuration")
        layers = []
        for i, L in enumerate(raw["layers"]):
            m = L["mixer"]
            if L["type"] == "parallel":
                a, r = m["left"], m["right"]
                rot = r.get("rot") or {}
                left = WindowSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a.get("vdim", a["dim"])), float(a["scale"]),
                                  int(a["mask"]["size"]), int(a["bias_max"]))
                right = RetentionSpec(int(r["heads"]), int(r["dim"]), int(r.get("vdim", r["dim"])), tuple(float(d) for d in r["decay"]),
                                      int(rot.get("dims", r["dim"])), float(rot.get("base", 10000.0)))
                if left.heads % left.kv_heads:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if left.size < 1:
                    raise ValueError(f"layer {i}: the window holds at least the position itself")
                if len(right.decay) != right.heads or not all(0.0 <= d <= 1.0 for d in right.decay):
                    raise ValueError(f"layer {i}: one decay in [0, 1] per retention head")
                if right.rot_dims % 2 or right.rot_dims > right.dim:
                    raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
                mix: PairSpec | DeltaSpec = PairSpec(left, right)
            elif L["type"] == "delta":
                mix = DeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), int(m["conv"]))
                if mix.heads % mix.kv_heads:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if not 1 <= mix.conv <= 64:
                    raise ValueError(f"layer {i}: {mix.conv} convolution taps")
            else:
                raise ValueError(f"layer {i}: mixer type {L['type']!r} is not one of this design")
            layers.append(LayerSpec(mix, NunosunConfig._mlp(i, L.get("mlp"))))
        taps = int(raw["canon"]["taps"])
        if not 1 <= taps <= 64:
            raise ValueError(f"canon.taps {taps}")
        return NunosunConfig(int(raw["vocab"]), int(raw["width"]), float(raw["norm"]["eps"]), int(raw["token_side"]["dim"]), taps,
                             float(raw.get("logit_scale", 1.0)), layers)

    @staticmethod
    def _mlp(i: int, mlp: dict | None) -> DenseSpec | ExpertsSpec | None:
        if not mlp:
            return None
        kind = mlp.get("kind", "dense")
        if kind == "dense":
            return DenseSpec(int(mlp["ff"]))
        if kind != "moe":
            raise ValueError(f"layer {i}: feed-forward kind {kind!r} is not one of this design")
        out = ExpertsSpec(int(mlp["expert"]["ff"]), int(mlp["router"]["experts"]), int(mlp["router"]["top"]))
        if not 0 < out.top <= out.experts <= 1024:
            raise ValueError(f"layer {i}: {out.top} of {out.experts} experts")
        return out

    def to_json(self) -> dict:
        out: dict = {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                     "canon": {"taps": self.taps}, "token_side": {"dim": self.side}, "logit_scale": self.logit_scale, "layers": []}
        for L in self.layers:
            m, f = L.mixer, L.mlp
            if isinstance(m, PairSpec):
                a, r = m.left, m.right
                kind, mix = "parallel", {
                    "left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                             "mask": {"size": a.size}, "bias_max": a.reach},
                    "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay),
                              "rot": {"dims": r.rot_dims, "base": r.rot_base}}}
            else:
                kind, mix = "delta", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
            mlp = None
            if isinstance(f, DenseSpec):
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            out["layers"].append({"type": kind, "mixer": mix, "mlp": mlp})
        return out

    def tensor_shapes(self) -> dict[str, tuple[int | None, ...]]:
        """Every checkpoint tensor by name (None: a size that only the checkpoint knows)."""
        w = self.width
        out: dict[str, tuple[int | None, ...]] = {
            "embed": (self.vocab, w), "embed.norm": (w,), "side.embed": (self.vocab, len(self.layers) * self.side),
            "head": (self.vocab, w), "final.norm": (w,)}
        for i, L in enumerate(self.layers):
            m, f, p = L.mixer, L.mlp, f"l{i}."
            x, y = p + "mix.", p + "mlp."
            out.update({p + "norm1": (w,), p + "canon1": (w, self.taps), p + "side.gate": (self.side, w), p + "side.proj": (w, self.side),
                        p + "side.norm": (w,)})
            if isinstance(m, PairSpec):
                a, r = m.left, m.right
                hd, hv = r.heads * r.dim, r.heads * r.vdim
                out.update({x + "left.q": (a.heads * a.dim, w), x + "left.k": (a.kv_heads * a.dim, w), x + "left.v": (a.kv_heads * a.vdim, w),
                            x + "left.q.norm": (a.dim,), x + "left.k.norm": (a.dim,), x + "left.rel": (a.buckets, a.heads),
                            x + "left.o": (w, a.heads * a.vdim), x + "left.out": (w,),
                            x + "right.q": (hd, w), x + "right.k": (hd, w), x + "right.v": (hv, w), x + "right.g": (hv, w),
                            x + "right.o": (w, hv), x + "right.out": (w,)})
            else:
                gd, hv = m.kv_heads * m.dim, m.heads * m.vdim
                for n, rows in (("q", gd), ("k", gd), ("v", hv)):
                    out.update({x + n: (rows, w), f"{x}{n}.conv": (rows, m.conv)})
                out.update({x + "g": (hv, w), x + "a": (m.heads, w), x + "b": (m.heads, w), x + "A_log": (m.heads,), x + "dt_bias": (m.heads,),
                            x + "norm": (m.vdim,), x + "o": (w, hv)})
            if isinstance(f, DenseSpec):
                out.update({y + "up": (f.ff, w), y + "down": (w, f.ff), y + "act": (4,)})
            elif f is not None:
                for j in range(f.experts):
                    out.update({f"{y}e{j}.gate": (f.ff, w), f"{y}e{j}.up": (f.ff, w), f"{y}e{j}.down": (w, f.ff)})
                out.update({y + "router": (f.experts, w), y + "router.b": (f.experts,)})
        return out

    @staticmethod
    def pattern(kinds: str, width: int, heads: int, kv_heads: int, dim: int, vdim: int, size: int, ret_heads: int, ret_dim: int, ret_vdim: int,
                delta_heads: int, delta_kv: int, delta_dim: int, delta_vdim: int, ff: int, expert_ff: int, experts: int, top: int, side: int,
                vocab: int, buckets: int = 32) -> "NunosunConfig":
        """Layers by letter (benchmarks, examples): ``d`` the delta rule with a dense feed-forward, ``p`` the pair with experts."""
        out = []
        for c in kinds:
            if c == "d":
                out.append(LayerSpec(DeltaSpec(delta_heads, delta_kv, delta_dim, delta_vdim, 4), DenseSpec(ff)))
            else:
                fixed = tuple(1.0 - 2.0 ** (-4.0 - 5.0 * h / max(1, ret_heads - 1)) for h in range(ret_heads))
                out.append(LayerSpec(PairSpec(WindowSpec(heads, kv_heads, dim, vdim, dim ** -0.5, size, max(2 * buckets, size), buckets),
                                              RetentionSpec(ret_heads, ret_dim, ret_vdim, fixed, ret_dim, 10000.0)),
                                     ExpertsSpec(expert_ff, experts, top)))
        return NunosunConfig(vocab, width, 1e-5, side, 4, 1.0, out)

    @staticmethod
    def tiny() -> "NunosunConfig":
        return NunosunConfig.pattern("dpd", 160, 4, 2, 32, 48, 100, 3, 48, 32, 4, 2, 48, 32, 320, 48, 6, 2, 20, 512, 24)


def synth_state(cfg: NunosunConfig, seed: int = 0, device="cpu") -> Iterator[tuple[str, torch.Tensor]]:
    """Seeded random checkpoint tensors (bf16): projections at 1/sqrt(fan-in), norms near 1, decays spread over short and long
    memories."""
    gen = torch.Generator(device=device)
    for idx, (name, shape) in enumerate(cfg.tensor_shapes().items()):
        shape = tuple(32 if n is None else n for n in shape)
        gen.manual_seed(seed * 1_000_003 + idx)
        r = torch.randn(shape, generator=gen, device=device)
        last = name.split(".")[-1]
        if "norm" in last or last == "out":
            t = 1.0 + 0.1 * r
        elif last == "A_log":
            t = 0.7 * r
        elif last == "dt_bias":
            t = -3.0 + 1.5 * r
        elif last == "canon1":
            t = 0.5 * r / math.sqrt(shape[1])
        elif last == "conv":
            t = r / math.sqrt(shape[1])
        elif last == "act":
            t = torch.tensor([0.6, 0.3, 0.2, 0.1], device=device) + 0.1 * r
        elif last == "rel" or name.endswith("router.b"):
            t = 0.5 * r
        elif name in ("embed", "side.embed"):
            t = r
        else:
            t = r / math.sqrt(shape[-1])
        yield name, t.bfloat16()


def write_checkpoint(directory: str, cfg: NunosunConfig, seed: int = 0) -> None:
    """config.json + model.safetensors with random weights."""
    from ..formats import safetensors_io
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg.to_json(), f, indent=1)
    safetensors_io.write_file(os.path.join(directory, "model.safetensors"), dict(synth_state(cfg, seed)))


# ---------------------------------------------------------------------------------------------- weights
@dataclass
class PairWeights:
    left: WindowAttention
    right: Retention
    proj: Projection                  # rows [left q | k | v | right q | k | v | gate]
    right_off: int
    left_o: Projection
    right_o: Projection
    left_w: torch.Tensor              # fp32 [ld]: norm weights with the factor of the mean in them
    right_w: torch.Tensor


@dataclass
class DeltaWeights:
    m: DeltaRule
    proj: Projection                  # rows [q | k | v | gate | a | b]
    o: Projection


@dataclass
class DenseWeights:
    ff: int
    up: Projection
    down: Projection
    act: tuple[float, float, float, float]


@dataclass
class ExpertsWeights:
    spec: ExpertsSpec
    router: Projection
    router_b: torch.Tensor            # fp32 [experts]
    w13: moe.ExpertWeights
    w2: moe.ExpertWeights


@dataclass
class NunosunLayer:
    mix: PairWeights | DeltaWeights
    norm: torch.Tensor                # fp32 [ld]
    conv: torch.Tensor                # fp32 [taps, ld], with the 1 of the row itself in the last tap
    side_gate: Projection
    side_proj: Projection
    side_norm: torch.Tensor
    ff: DenseWeights | ExpertsWeights | None = None


def _fits(have: tuple[int, ...], want: tuple[int | None, ...]) -> bool:
    return len(have) == len(want) and all(w is None or h == w for h, w in zip(have, want))


class NunosunWeights:
    """Device-resident, padded, kernel-ready weights from (name, tensor) pairs."""

    def __init__(self, cfg: NunosunConfig, state, device="cuda", dtype: torch.dtype = torch.bfloat16):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("activations are bfloat16 or float32")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        t = dict(state)
        shapes = cfg.tensor_shapes()
        missing = [n for n in shapes if n not in t]
        wrong = [f"{n} {tuple(t[n].shape)} != {s}" for n, s in shapes.items() if n in t and not _fits(tuple(t[n].shape), s)]
        if missing or wrong:                       # tensors the configuration does not mention are left unread
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:4]}, shapes {wrong[:4]}")
        self.ld, self.side = pad16(cfg.width), pad16(cfg.side)
        self.embed = torch.zeros(cfg.vocab, self.ld, dtype=dtype, device=self.device)
        self.embed[:, :cfg.width] = t["embed"].to(self.device, dtype)
        self.embed_norm = self._row(t["embed.norm"])
        self.side_embed = torch.zeros(cfg.vocab, len(cfg.layers), self.side, dtype=dtype, device=self.device)
        self.side_embed[:, :, :cfg.side] = t["side.embed"].to(self.device, dtype).view(cfg.vocab, len(cfg.layers), cfg.side)
        self.side_embed = self.side_embed.view(cfg.vocab, -1)
        self.head = self._proj(t["head"], pad_n=False)
        self.final_norm = self._row(t["final.norm"], scale=cfg.logit_scale)
        self.head_lo = 0
        self.layers: list[NunosunLayer] = []
        for i, L in enumerate(cfg.layers):
            p = f"l{i}."
            sub = lambda what: {n[len(p) + len(what) + 1:]: v for n, v in t.items() if n.startswith(p + what + ".")}
            mix = self._pair(L.mixer, sub("mix")) if isinstance(L.mixer, PairSpec) else self._delta(L.mixer, sub("mix"))
            conv = torch.zeros(cfg.taps, self.ld, dtype=torch.float32, device=self.device)
            conv[:, :cfg.width] = t[p + "canon1"].to(self.device, torch.float32).t()
            conv[-1, :cfg.width] += 1.0
            ff = None
            if isinstance(L.mlp, DenseSpec):
                ff = self._dense(L.mlp, sub("mlp"))
            elif L.mlp is not None:
                ff = self._experts(L.mlp, sub("mlp"))
            self.layers.append(NunosunLayer(mix, self._row(t[p + "norm1"]), conv, self._proj(t[p + "side.gate"]), self._proj(t[p + "side.proj"]),
                                            self._row(t[p + "side.norm"]), ff))

    def _proj(self, w: torch.Tensor, pad_n: bool = True, tile_n: bool = False) -> Projection:
        return Projection.make(w, self.dtype, self.device, pad_n, tile_n)

    def _row(self, w: torch.Tensor, n: int | None = None, scale: float = 1.0) -> torch.Tensor:
        """fp32 row padded with zeros to n (default: the residual's width)."""
        out = torch.zeros(n or self.ld, dtype=torch.float32, device=self.device)
        out[:w.numel()] = w.reshape(-1).to(self.device, torch.float32) * scale
        return out

    def _pair(self, s: PairSpec, t: dict[str, torch.Tensor]) -> PairWeights:
        a, r = s.left, s.right
        d, v, rd, rv = (pad16(n) for n in (a.dim, a.vdim, r.dim, r.vdim))
        rel = t["left.rel"]
        if rel.shape[0] < 2 or not a.reach > rel.shape[0] // 2:
            raise ValueError("the distance bias needs two rows and a reach beyond half of them")
        if max(d, v) > 1024 or rd > 512:
            raise ValueError("attention heads up to 1024 values and retention heads up to 512 key channels")
        left = WindowAttention(a.heads, a.kv_heads, a.dim, d, a.vdim, v, a.scale, a.size, self.cfg.eps, self._row(t["left.q.norm"], d),
                               self._row(t["left.k.norm"], d), winattn.distance_bias(rel.to(self.device), a.size, a.reach))
        freq = r.rot_base ** (-torch.arange(0, r.rot_dims, 2, dtype=torch.float64) / max(r.rot_dims, 1))
        fixed = torch.tensor(r.decay, dtype=torch.float64)
        right = Retention(r.heads, r.dim, rd, r.vdim, rv, self.cfg.eps, r.rot_dims, freq.to(self.device), fixed.float().to(self.device),
                          torch.log2(fixed).float().to(self.device), torch.ones(rv, dtype=torch.float32, device=self.device))
        rows = [(pad_heads(t["left." + n], h, ((real, pad),)), h * pad)
                for n, h, real, pad in (("q", a.heads, a.dim, d), ("k", a.kv_heads, a.dim, d), ("v", a.kv_heads, a.vdim, v))]
        off = sum(n for _, n in rows)
        rows += [(pad_heads(t["right." + n], r.heads, ((real, pad),)), r.heads * pad)
                 for n, real, pad in (("q", r.dim, rd), ("k", r.dim, rd), ("v", r.vdim, rv), ("g", r.vdim, rv))]
        back = lambda w, h, real, pad: self._proj(pad_heads(w.t().contiguous(), h, ((real, pad),)).t())
        return PairWeights(left, right, self._proj(cat_rows(rows), tile_n=True), off, back(t["left.o"], a.heads, a.vdim, v),
                           back(t["right.o"], r.heads, r.vdim, rv), self._row(t["left.out"], scale=0.5), self._row(t["right.out"], scale=0.5))

    def _delta(self, s: DeltaSpec, t: dict[str, torch.Tensor]) -> DeltaWeights:
        d, v = pad16(s.dim), pad16(s.vdim)
        if d > 512 or v > 2048:
            raise ValueError("the delta rule takes up to 512 key and 2048 value channels per head")
        keys = lambda n: pad_heads(t[n], s.kv_heads, ((s.dim, d),))
        values = lambda n: pad_heads(t[n], s.heads, ((s.vdim, v),))
        conv = torch.cat([keys("q.conv"), keys("k.conv"), values("v.conv")]).to(self.device, torch.float32).t().contiguous()
        m = DeltaRule(s.heads, s.kv_heads, s.dim, d, s.vdim, v, self.cfg.eps, conv,
                      -torch.exp(t["A_log"].to(self.device).double()).float(), self._row(t["dt_bias"], s.heads), self._row(t["norm"], v))
        rows = [keys("q"), keys("k"), values("v"), values("g"), t["a"], t["b"]]
        return DeltaWeights(m, self._proj(torch.cat(rows), tile_n=True),
                            self._proj(pad_heads(t["o"].t().contiguous(), s.heads, ((s.vdim, v),)).t()))

    def _dense(self, f: DenseSpec, t: dict[str, torch.Tensor]) -> DenseWeights:
        return DenseWeights(f.ff, self._proj(t["up"], tile_n=True), self._proj(t["down"]), tuple(float(x) for x in t["act"]))

    def _experts(self, f: ExpertsSpec, t: dict[str, torch.Tensor]) -> ExpertsWeights:
        w13, w2 = moe.pack_experts(*([t[f"e{j}.{n}"] for j in range(f.experts)] for n in ("gate", "up", "down")), self.cfg.width, self.ld,
                                   self.dtype, self.device)
        return ExpertsWeights(f, self._proj(t["router"]), self._row(t["router.b"], f.experts), w13, w2)

    def nbytes(self) -> int:
        size = lambda x: x.numel() * x.element_size()
        n = size(self.embed) + size(self.side_embed) + self.head.nbytes()
        for L in self.layers:
            m = L.mix
            own = (m.proj, m.left_o, m.right_o) if isinstance(m, PairWeights) else (m.proj, m.o)
            n += sum(p.nbytes() for p in (*own, L.side_gate, L.side_proj))
            if isinstance(L.ff, DenseWeights):
                n += L.ff.up.nbytes() + L.ff.down.nbytes()
            elif L.ff is not None:
                n += L.ff.router.nbytes() + size(L.ff.w13.weight) + size(L.ff.w2.weight)
        return n


# ---------------------------------------------------------------------------------------------- runtime
class NunosunRuntime(PagedRuntime):
    exposes_logits = True
    tile_min_rows = winattn.TILE_MIN_ROWS

    def __init__(self, cfg: NunosunConfig, weights: NunosunWeights, max_slots: int = 1, max_context: int = 4096,
                 block_size: int = 64, num_blocks: int | None = None, comm=None):
        super().__init__(weights.device, max_slots, max_context, block_size, num_blocks, comm)
        if self.comm.world != 1:
            raise ValueError("a Nunosun model runs on one rank")
        self.cfg, self.w = cfg, weights
        tiles = weights.dtype == torch.bfloat16 and all(winattn.tiles_supported(lw.mix.left, block_size) for lw in weights.layers
                                                        if isinstance(lw.mix, PairWeights))
        if not tiles:
            self.tile_min_rows = 1 << 30              # every row on the row kernel (fp32, or heads wider than the tile kernel takes)
        self.window = max([L.mixer.left.size for L in cfg.layers if isinstance(L.mixer, PairSpec)], default=0)
        self.k_cache: list[torch.Tensor | None] = []
        self.v_cache: list[torch.Tensor | None] = []
        self.state: list[torch.Tensor] = []
        self.conv_tail: list[torch.Tensor | None] = []
        self.row_tail: list[torch.Tensor] = []        # last inputs of the convolution in front of the mixer
        pages = lambda width, what: canary.zeros(self.num_blocks, block_size, width, dtype=weights.dtype, device=self.device, name=what)
        for i, (L, lw) in enumerate(zip(cfg.layers, weights.layers)):
            k = v = tail = None
            if isinstance(lw.mix, PairWeights):
                m = lw.mix.right
                k, v = pages(lw.mix.left.k_width, f"paged key cache of layer {i}"), pages(lw.mix.left.v_width, f"paged value cache of layer {i}")
            else:
                m = lw.mix.m
                tail = self.slot_state(max(L.mixer.conv - 1, 1), m.channels, dtype=weights.dtype, name=f"convolution tail of layer {i}")
            self.k_cache.append(k)
            self.v_cache.append(v)
            self.conv_tail.append(tail)
            self.state.append(self.slot_state(m.heads, m.d, m.v, dtype=torch.float32, name=f"recurrent state of layer {i}"))
            self.row_tail.append(self.slot_state(max(cfg.taps - 1, 1), weights.ld, dtype=weights.dtype, name=f"row tail of layer {i}"))
        self._side_stream: torch.cuda.Stream | None = None
        self.residual_tap = None                      # debugging: called with (layer, residual [T, width]) after every layer

    def history_floor(self, length: int) -> int:
        return max(0, length - max(self.window - 1, 0))

    def history_span(self) -> int | None:
        return max(self.window - 1, 0)

    def _pair(self, i: int, pw: PairWeights, y: torch.Tensor, positions, kv_slots, meta):
        m, k, v, t = pw.left, self.k_cache[i], self.v_cache[i], y.shape[0]
        proj = pw.proj(y)
        q = winattn.head_prep(proj, m, positions, kv_slots, k, v)
        out = torch.empty(t, pw.left_o.k, dtype=y.dtype, device=y.device)
        n = meta["tile_rows"] if meta["mode"] == "mixed" else 0
        if n:
            winattn.prefill(q[:n], m, k, v, self.block_table, meta["q_start"], meta["q_len"], meta["kv_len"], meta["max_q_len"], out[:n],
                            seq=meta["tile_seq"])
        if meta["mode"] == "decode":
            winattn.rows(q, m, k, v, meta["block_table"], positions, meta["max_kv_len"], out)
        elif n < t:
            winattn.rows(q[n:], m, k, v, self.block_table, positions[n:], meta["max_kv_len"], out[n:], seq=meta["row_seq"][n:])
        left = pw.left_o(out)
        right = pw.right_o(decay.retention(proj[:, pw.right_off:], pw.right, self.state[i], meta["segments"], positions, pw.right_o.k))
        return (left, pw.left_w), (right, pw.right_w)

    def _experts(self, ew: ExpertsWeights, h: torch.Tensor) -> Routed:
        f = ew.spec
        idx, weights = moe.route(moe.router_logits(h, ew.router)[:, :f.experts], ew.router_b, f.top, "softmax_chosen", True, 1.0)
        y, row = moe.experts_rows(h, idx, ew.w13, ew.w2)
        return Routed(y, row, idx, weights, f.experts)

    def _feed_forward(self, ff: DenseWeights | ExpertsWeights, h: torch.Tensor) -> dict:
        if isinstance(ff, DenseWeights):
            return {"dense": ff.down(decoder.poly_norm(ff.up(h), ff.ff, ff.act, self.cfg.eps, ff.down.k))}
        return {"routed": self._experts(ff, h)}

    @contextlib.contextmanager
    def _beside(self, on: bool):
        """Work inside runs on a second stream, beside what the caller launches until it leaves ``join`` (yielded) behind.
        Tensors made inside are read after the join only, and the next work on that stream waits for those readers."""
        if not on:
            yield lambda: None
            return
        if self._side_stream is None:
            self._side_stream = torch.cuda.Stream(self.device)
        main, side = torch.cuda.current_stream(self.device), self._side_stream
        side.wait_event(main.record_event())
        with torch.cuda.stream(side), gemm.scratch(1):
            yield lambda: main.wait_event(side.record_event())

    def _forward(self, ids, positions, kv_slots, meta, rows):
        cfg, w, n = self.cfg, self.w, ids.numel()
        x = torch.empty(n, w.ld, dtype=torch.float32, device=self.device)
        common = {"ld": w.ld, "n": n, "dtype": w.dtype}
        exact = w.dtype == torch.float32
        pending: dict = {"ids": ids, "table": w.embed, "normed": ((None, w.embed_norm),)}       # the residual starts from it

        def step(**kw):
            """What is pending enters the residual."""
            nonlocal pending
            out = decoder.branch_step(None if "ids" in pending else x, cfg.width, cfg.eps, **common, **pending, **kw)
            pending = {}
            return out

        for i, lw in enumerate(w.layers):
            _, h, m = step(x_out=x, weight=lw.norm, conv=lw.conv, tail=self.row_tail[i], seg=meta["segments"], positions=positions)
            # a decoding step is bound by launches and by the weights' stream: the sublayers run beside each other
            join, extra = lambda: None, {}
            if lw.ff is not None:
                with self._beside(meta["mode"] == "decode") as join:
                    extra = self._feed_forward(lw.ff, h)
            if isinstance(lw.mix, PairWeights):
                pending = {"normed": self._pair(i, lw.mix, m, positions, kv_slots, meta), "plain": ()}
            else:
                d = lw.mix
                y = d.o(decay.delta_rule(d.proj(m), d.m, self.state[i], self.conv_tail[i], meta["segments"], positions, d.o.k))
                pending = {"plain": (y,)}
            join()
            if "dense" in extra:
                pending["plain"] += (extra["dense"],)
            pending["routed"] = extra.get("routed")
            c = step(x_out=x, copy=not exact)[0]
            g = decoder.token_gate(x if exact else c, lw.side_gate, w.side_embed, i * w.side, ids)
            pending = {"normed": ((lw.side_proj(g), lw.side_norm),)}
            if self.residual_tap is not None:
                step(x_out=x)
                self.residual_tap(i, x[:, :cfg.width].clone())
        if rows is not None and rows.numel() == 0:
            return None
        return w.head(step(weight=w.final_norm, rows=rows)[1], out_f32=True)


def build_synthetic(cfg: NunosunConfig, device="cuda", seed: int = 0, dtype: torch.dtype = torch.bfloat16, **kw) -> NunosunRuntime:
    """Random-weight runtime of the given shape."""
    return NunosunRuntime(cfg, NunosunWeights(cfg, synth_state(cfg, seed, device), device, dtype), **kw)
