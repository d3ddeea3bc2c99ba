"""Rutulix decoder: attention whose scores are mixed across heads (values are the raw key projection, whole-row QK norm,
interleaved rotary with YaRN, attention inside fixed chunks of positions), a dense feed-forward with biases and the xIELU
activation, layer norms before and after each sublayer, an fp32 residual, and a run of layers that is repeated with the
same weights.

The layers are described by config.json (sizes, order, constants); the passes, the pages and the batching come from
``models/paged.py``, the kernels from ``ops/mixattn.py``.  Activations are bf16 (serving) or fp32 (``dtype``).
A looped layer has one cache per pass.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Iterator

import torch

from ..ops import mixattn
from ..ops.mixattn import HeadMix, Projection, pad8, pad16
from ..utils import canary
from .paged import PagedRuntime

ARCH = "Rutulix"
# kernel sources the runtime launches (a partial build compiles only these)
KERNEL_SOURCES = ("residual_norm.cu", "bias_act.cu", "qk_row_prep.cu", "attn_mix_rows.cu", "attn_mix_prefill.cu", "gemm_f32.cu",
                  "gemm_wdec.cu", "gemm_bf16_2cta.cu", "elementwise.cu", "sampling.cu", "bounds.cu")


# ---------------------------------------------------------------------------------------------- configuration
@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    chunk: int = 0                    # 0: plain causal
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_scaling: dict | None = None


@dataclass
class LayerSpec:
    mixer: AttentionSpec
    ff: int = 0                       # 0: no feed-forward


@dataclass
class RutulixConfig:
    vocab: int
    width: int
    eps: float
    layers: list[LayerSpec] = field(default_factory=list)
    loop: tuple[int, int, int] | None = None        # (start, stop, times)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def is_rutulix_json(raw: Any) -> bool:
        return isinstance(raw, dict) and raw.get("architecture") == ARCH

    @staticmethod
    def from_json(raw: dict) -> "RutulixConfig":
        if not RutulixConfig.is_rutulix_json(raw):
            raise ValueError(f"not a {ARCH} configuration")
        layers = []
        for i, L in enumerate(raw["layers"]):
            if L["type"] != "attention":
                raise ValueError(f"layer {i}: mixer type {L['type']!r} is not one of this design")
            m = L["mixer"]
            if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                raise ValueError(f"layer {i}: the values are the keys, so vdim must equal dim")
            if int(m["heads"]) % int(m["kv_heads"]):
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            rot, mask, mlp = m.get("rot") or {}, m.get("mask") or {}, L.get("mlp")
            if int(rot.get("dims", 0)) % 2 or int(rot.get("dims", 0)) > int(m["dim"]):
                raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not one of this design")
            layers.append(LayerSpec(AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), float(m["scale"]),
                                                  int(mask.get("size") or 0), int(rot.get("dims", 0)),
                                                  float(rot.get("base", 10000.0)), rot.get("scaling")),
                                    int(mlp["ff"]) if mlp else 0))
        lp = raw.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
        if loop and not (0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
            raise ValueError(f"loop {lp} does not fit {len(layers)} layers")
        return RutulixConfig(int(raw["vocab"]), int(raw["width"]), float(raw["norm"]["eps"]), layers, loop)

    def to_json(self) -> dict:
        out: dict = {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": []}
        for L in self.layers:
            a = L.mixer
            mix: dict = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.dim, "scale": a.scale}
            if a.chunk:
                mix["mask"] = {"size": a.chunk}
            if a.rot_dims:
                mix["rot"] = {"dims": a.rot_dims, "base": a.rot_base}
                if a.rot_scaling:
                    mix["rot"]["scaling"] = dict(a.rot_scaling)
            out["layers"].append({"type": "attention", "mixer": mix, "mlp": {"kind": "dense", "ff": L.ff} if L.ff else None})
        if self.loop:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def runs(self) -> list[tuple[int, int | None]]:
        """(layer, number of the pass that begins right before it, or None) in execution order."""
        n = len(self.layers)
        if not self.loop:
            return [(i, None) for i in range(n)]
        a, b, times = self.loop
        passes = [(i, t if i == a else None) for t in range(times) for i in range(a, b)]
        return [(i, None) for i in range(a)] + passes + [(i, None) for i in range(b, n)]

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every checkpoint tensor by name."""
        w = self.width
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab, w), "head": (self.vocab, w), "final.norm": (w,)}
        if self.loop:
            out["loop.step"] = (self.loop[2], w)
        for i, L in enumerate(self.layers):
            a, p = L.mixer, f"l{i}."
            qn, kn = a.heads * a.dim, a.kv_heads * a.dim
            out.update({p + "norm1": (w,), p + "norm1b": (w,), p + "mix.q": (qn, w), p + "mix.k": (kn, w),
                        p + "mix.q.norm": (qn,), p + "mix.k.norm": (kn,), p + "mix.talk": (a.heads, a.heads),
                        p + "mix.o": (w, qn)})
            if L.ff:
                out.update({p + "norm2": (w,), p + "norm2b": (w,), p + "mlp.up": (L.ff, w), p + "mlp.up.b": (L.ff,),
                            p + "mlp.down": (w, L.ff), p + "mlp.down.b": (w,), p + "mlp.act": (2,)})
        return out

    @staticmethod
    def uniform(layers: int, width: int, heads: int, kv_heads: int, dim: int, ff: int, vocab: int, chunk: int,
                loop: tuple[int, int, int] | None = None, rot_dims: int | None = None) -> "RutulixConfig":
        """Equal layers throughout (benchmarks, examples)."""
        a = AttentionSpec(heads, kv_heads, dim, dim ** -0.5, chunk, dim // 2 if rot_dims is None else rot_dims, 500000.0,
                          {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0})
        return RutulixConfig(vocab, width, 1e-5, [LayerSpec(a, ff) for _ in range(layers)], loop)

    @staticmethod
    def tiny() -> "RutulixConfig":
        return RutulixConfig.uniform(3, 192, 6, 3, 32, 320, 512, 48, loop=(0, 2, 2))


def synth_state(cfg: RutulixConfig, seed: int = 0, device="cpu") -> Iterator[tuple[str, torch.Tensor]]:
    """Seeded random checkpoint tensors (bf16): projections at 1/sqrt(fan-in), norms near 1, a mixing matrix near the
    identity."""
    gen = torch.Generator(device=device)
    for idx, (name, shape) in enumerate(cfg.tensor_shapes().items()):
        gen.manual_seed(seed * 1_000_003 + idx)
        r = torch.randn(shape, generator=gen, device=device)
        if "norm" in name.split(".")[-1]:
            t = 1.0 + 0.1 * r
        elif name.endswith(".talk"):
            t = torch.eye(shape[0], device=device) + 0.3 * r
        elif name.endswith(".b") or name == "loop.step":
            t = 0.2 * r
        elif name.endswith(".act"):
            t = 0.5 * r
        elif name == "embed":
            t = r
        else:
            t = r / math.sqrt(shape[-1])
        yield name, t.bfloat16()


def write_checkpoint(directory: str, cfg: RutulixConfig, seed: int = 0) -> None:
    """config.json + model.safetensors with random weights."""
    from ..formats import safetensors_io
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg.to_json(), f, indent=1)
    safetensors_io.write_file(os.path.join(directory, "model.safetensors"), dict(synth_state(cfg, seed)))


# ---------------------------------------------------------------------------------------------- weights
@dataclass
class RutulixLayer:
    mix: HeadMix
    norm1: torch.Tensor
    norm1b: torch.Tensor
    qk: Projection                    # rows [query heads | key heads], heads padded to mix.d
    o: Projection
    norm2: torch.Tensor | None = None
    norm2b: torch.Tensor | None = None
    up: Projection | None = None
    up_b: torch.Tensor | None = None
    down: Projection | None = None
    down_b: torch.Tensor | None = None
    act: tuple[float, float] = (0.0, 0.0)


class RutulixWeights:
    """Device-resident, padded, kernel-ready weights from (name, tensor) pairs."""

    def __init__(self, cfg: RutulixConfig, state, device="cuda", dtype: torch.dtype = torch.bfloat16):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("activations are bfloat16 or float32")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        t = dict(state)
        shapes = cfg.tensor_shapes()
        missing = [n for n in shapes if n not in t]
        wrong = [f"{n} {tuple(t[n].shape)} != {s}" for n, s in shapes.items() if n in t and tuple(t[n].shape) != s]
        if missing or wrong:                       # tensors the configuration does not mention are left unread
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:4]}, shapes {wrong[:4]}")
        dev, self.ld = self.device, pad16(cfg.width)
        proj = lambda w, pad_n=True: Projection.make(w, dtype, dev, pad_n)

        def row(w: torch.Tensor, n: int | None = None) -> torch.Tensor:
            """fp32 row padded with zeros to n (default: the residual's width)."""
            out = torch.zeros(n or self.ld, dtype=torch.float32, device=dev)
            out[:w.numel()] = w.to(dev, torch.float32)
            return out

        self.embed = torch.zeros(cfg.vocab, self.ld, dtype=dtype, device=dev)
        self.embed[:, :cfg.width] = t["embed"].to(dev, dtype)
        self.head = proj(t["head"], False)
        self.final_norm = row(t["final.norm"])
        self.steps = [row(s) for s in t["loop.step"]] if cfg.loop else []
        self.head_lo = 0
        self.layers: list[RutulixLayer] = []
        for i, L in enumerate(cfg.layers):
            a, p = L.mixer, f"l{i}."
            d = pad8(a.dim)

            def heads(w: torch.Tensor, n: int) -> torch.Tensor:
                """[n * dim, ...] -> [n * d, ...]: zero rows after every head."""
                out = torch.zeros(n, d, *w.shape[1:], dtype=w.dtype, device=w.device)
                out[:, :a.dim] = w.reshape(n, a.dim, *w.shape[1:])
                return out.reshape(n * d, *w.shape[1:])

            freq, mscale = mixattn.yarn_freqs(a.rot_dims, a.rot_base, a.rot_scaling, dev)
            talk_t = torch.zeros(a.heads, (a.heads + 3) // 4 * 4, dtype=torch.float32, device=dev)
            talk_t[:, :a.heads] = t[p + "mix.talk"].to(dev, torch.float32).t()
            mix = HeadMix(a.heads, a.kv_heads, a.dim, d, a.scale, a.chunk, a.rot_dims, freq, mscale, cfg.eps,
                          heads(t[p + "mix.q.norm"].to(dev, torch.float32), a.heads).contiguous(),
                          heads(t[p + "mix.k.norm"].to(dev, torch.float32), a.kv_heads).contiguous(), talk_t)
            lw = RutulixLayer(mix, row(t[p + "norm1"]), row(t[p + "norm1b"]),
                              proj(torch.cat([heads(t[p + "mix.q"], a.heads), heads(t[p + "mix.k"], a.kv_heads)])),
                              proj(heads(t[p + "mix.o"].t().contiguous(), a.heads).t()))
            if L.ff:
                act = t[p + "mlp.act"].double().tolist()
                soft = lambda z: math.log1p(math.exp(-abs(z))) + max(z, 0.0)
                lw.norm2, lw.norm2b = row(t[p + "norm2"]), row(t[p + "norm2b"])
                lw.up, lw.up_b = proj(t[p + "mlp.up"]), row(t[p + "mlp.up.b"], pad16(L.ff))
                lw.down, lw.down_b = proj(t[p + "mlp.down"]), row(t[p + "mlp.down.b"])
                lw.act = (soft(act[0]), 0.5 + soft(act[1]))
            self.layers.append(lw)

    def nbytes(self) -> int:
        n = self.embed.numel() * self.embed.element_size() + self.head.nbytes()
        for L in self.layers:
            n += sum(p.nbytes() for p in (L.qk, L.o, L.up, L.down) if p is not None)
        return n


# ---------------------------------------------------------------------------------------------- runtime
class RutulixRuntime(PagedRuntime):
    exposes_logits = True
    tile_min_rows = mixattn.TILE_MIN_ROWS

    def __init__(self, cfg: RutulixConfig, weights: RutulixWeights, max_slots: int = 1, max_context: int = 4096,
                 block_size: int = 64, num_blocks: int | None = None, comm=None):
        super().__init__(weights.device, max_slots, max_context, block_size, num_blocks, comm)
        if self.comm.world != 1:
            raise ValueError("the scores of all heads are mixed: the model runs on one rank")
        self.cfg, self.w = cfg, weights
        self.runs = cfg.runs()
        self.chunks = [L.mixer.chunk for L in cfg.layers]
        self.k_cache, self.v_cache = [], []
        for r, (li, _) in enumerate(self.runs):
            m = weights.layers[li].mix
            for store, name in ((self.k_cache, "key"), (self.v_cache, "value")):
                store.append(canary.zeros(self.num_blocks, block_size, m.groups * m.d, dtype=weights.dtype, device=self.device,
                                          name=f"paged {name} cache of layer run {r}"))
        tiles = weights.dtype == torch.bfloat16 and all(mixattn.tiles_supported(L.mix, block_size) for L in weights.layers)
        if not tiles:
            self.tile_min_rows = 1 << 30          # every row on the row kernel (fp32, or heads wider than the tile kernel takes)
        self.residual_tap = None                  # debugging: called with (layer run, residual [T, width]) after every layer run

    def history_floor(self, length: int) -> int:
        return min((length - length % c if c else 0) for c in self.chunks) if self.chunks else 0

    def history_span(self) -> int | None:
        return max(self.chunks) - 1 if self.chunks and all(self.chunks) else None

    def _attention(self, run: int, lw: RutulixLayer, y: torch.Tensor, positions, kv_slots, meta) -> torch.Tensor:
        m, k, v = lw.mix, self.k_cache[run], self.v_cache[run]
        t = y.shape[0]
        n = meta["tile_rows"] if meta["mode"] == "mixed" else 0
        q_mix, q_row = mixattn.qk_row_prep(lw.qk(y), m, positions, kv_slots, k, v, n)
        ldo = lw.o.k
        out = (torch.empty if ldo == m.heads * m.d else torch.zeros)(t, ldo, dtype=y.dtype, device=y.device)
        if n:
            mixattn.prefill(q_mix, m, k, v, self.block_table, meta["q_start"], meta["q_len"], meta["kv_len"], meta["max_q_len"],
                            out[:n], seq=meta["tile_seq"])
        if n < t:
            keys = min(meta["max_kv_len"], m.chunk) if m.chunk else meta["max_kv_len"]
            if meta["mode"] == "decode":
                mixattn.rows(q_row, m, k, v, meta["block_table"], positions, keys, out)
            else:
                mixattn.rows(q_row, m, k, v, self.block_table, positions[n:], keys, out[n:], seq=meta["row_seq"][n:])
        return lw.o(out)

    def _mlp(self, lw: RutulixLayer, y: torch.Tensor) -> torch.Tensor:
        return lw.down(lw.up.bias_xielu(y, lw.up_b, *lw.act))

    def _forward(self, ids, positions, kv_slots, meta, rows):
        cfg, w = self.cfg, self.w
        x = torch.empty(ids.numel(), w.ld, dtype=torch.float32, device=self.device)
        src = {"ids": ids, "table": w.embed}                   # the first boundary starts the residual
        pending: dict = {}                                     # sublayer output that has not entered the residual yet

        def boundary(**kw):
            nonlocal src, pending
            out = mixattn.residual_norm(x, cfg.width, cfg.eps, dtype=w.dtype, **src, **pending, **kw)
            src, pending = {}, {}
            return out

        for run, (li, begins) in enumerate(self.runs):
            lw = w.layers[li]
            y = boundary(step=None if begins is None else w.steps[begins], pre_w=lw.norm1)
            pending = {"delta": self._attention(run, lw, y, positions, kv_slots, meta), "post_w": lw.norm1b}
            if lw.up is not None:
                y = boundary(pre_w=lw.norm2)
                pending = {"delta": self._mlp(lw, y), "bias": lw.down_b, "post_w": lw.norm2b}
            if self.residual_tap is not None:
                boundary()
                self.residual_tap(run, x[:, :cfg.width].clone())
        if rows is not None and rows.numel() == 0:
            return None
        y = boundary(pre_w=w.final_norm, rows=rows)
        return w.head(y, out_f32=True)


def build_synthetic(cfg: RutulixConfig, device="cuda", seed: int = 0, dtype: torch.dtype = torch.bfloat16, **kw) -> RutulixRuntime:
    """Random-weight runtime of the given shape."""
    return RutulixRuntime(cfg, RutulixWeights(cfg, synth_state(cfg, seed, device), device, dtype), **kw)
