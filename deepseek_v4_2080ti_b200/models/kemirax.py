"""Kemirax decoder: layers whose mixer and feed-forward read one norm side by side, each result behind an element-wise sigmoid
gate.  Mixers are latent attention (low-rank queries, one cached latent and rotated key part per token for all heads; a layer
may read another layer's cache) and gated linear attention (a decay per key channel); what a mixer reads is moved towards the
previous token's row.  The feed-forward routes to small experts, some of which are the identity, beside a gated shared expert.

The layers are described by config.json (sizes, order, constants); the passes, the pages, the state slots and the batching
come from ``models/paged.py``, the kernels from ``ops/latent.py``, ``ops/gla.py``, ``ops/moe.py`` and ``ops/decoder.py``.
Activations are bf16 (serving) or fp32 (``dtype``).
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Iterator

import torch

from ..ops import decoder, gla, latent, moe
from ..ops.decoder import Projection, Routed, cat_rows, pad16, pad_heads
from ..ops.gemm import PackedLinear
from ..ops.gla import GatedLinear
from ..ops.latent import LatentAttention
from ..ops.mixattn import yarn_freqs
from ..utils import canary
from .paged import PagedRuntime

ARCH = "Kemirax"
UNIT_SLOPE = 1.702
SHORT_ROWS = 128              # batches up to this are bound by the weights' bytes and by launches
# kernel sources the runtime launches (a partial build compiles only these)
KERNEL_SOURCES = ("parallel_step.cu", "latent_prep.cu", "attn_latent_rows.cu", "attn_latent_decode.cu", "attn_heads_prefill.cu",
                  "head_linear.cu", "gated_linear.cu", "gla_chunk.cu", "moe.cu",
                  "bias_act.cu", "gemm_f32.cu", "gemm_wdec.cu", "gemm_bf16_2cta.cu", "elementwise.cu", "sampling.cu", "bounds.cu")


# ---------------------------------------------------------------------------------------------- configuration
@dataclass
class LatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_dims: int
    rot_base: float
    rot_scaling: dict | None = None
    kv_from: int | None = None        # reads this layer's cache


@dataclass
class LinearSpec:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int | None = None           # of the decay's low-rank projection; None: what the checkpoint's tensors have


@dataclass
class ExpertsSpec:
    ff: int
    limit: float
    experts: int
    identity: int
    top: int
    shared_ff: int = 0                # 0: no shared expert
    shared_limit: float = 0.0


@dataclass
class LayerSpec:
    mixer: LatentSpec | LinearSpec
    mlp: ExpertsSpec | None = None


@dataclass
class KemiraxConfig:
    vocab: int
    width: int
    eps: float
    layers: list[LayerSpec] = field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def is_kemirax_json(raw: Any) -> bool:
        return isinstance(raw, dict) and raw.get("architecture") == ARCH

    @staticmethod
    def from_json(raw: dict) -> "KemiraxConfig":
        if not KemiraxConfig.is_kemirax_json(raw):
            raise ValueError(f"not a {ARCH} configuration")
        layers: list[LayerSpec] = []
        for i, L in enumerate(raw["layers"]):
            m = L["mixer"]
            if L["type"] == "latent_attention":
                rot, src = m.get("rot") or {}, m.get("kv_from")
                rot_dim = int(m["rot_dim"])
                mix: LatentSpec | LinearSpec = LatentSpec(
                    int(m["heads"]), int(m["dim"]), rot_dim, int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]), float(m["scale"]),
                    int(rot.get("dims", rot_dim)), float(rot.get("base", 10000.0)), rot.get("scaling"), None if src is None else int(src))
                if mix.rot_dims % 2 or mix.rot_dims > rot_dim:
                    raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim")
                if src is not None:
                    o = layers[mix.kv_from].mixer if 0 <= mix.kv_from < i else None
                    if not isinstance(o, LatentSpec) or o.kv_from is not None or (o.kv_rank, o.rot_dim) != (mix.kv_rank, mix.rot_dim):
                        raise ValueError(f"layer {i}: kv_from {src} is not an earlier latent attention layer with an equal cache of its own")
            elif L["type"] == "gla":
                mix = LinearSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]),
                                 int(m["rank"]) if m.get("rank") is not None else None)
                if not mix.tau > 0:
                    raise ValueError(f"layer {i}: tau must be positive")
            else:
                raise ValueError(f"layer {i}: mixer type {L['type']!r} is not one of this design")
            layers.append(LayerSpec(mix, KemiraxConfig._mlp(i, L.get("mlp"))))
        return KemiraxConfig(int(raw["vocab"]), int(raw["width"]), float(raw["norm"]["eps"]), layers)

    @staticmethod
    def _mlp(i: int, mlp: dict | None) -> ExpertsSpec | None:
        if not mlp:
            return None
        if mlp.get("kind", "moe") != "moe":
            raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not one of this design")
        e, r, s = mlp["expert"], mlp["router"], mlp.get("shared") or {}
        out = ExpertsSpec(int(e["ff"]), float(e["limit"]), int(r["experts"]), int(r.get("identity") or 0), int(r["top"]),
                          int(s.get("ff", 0)), float(s.get("limit", 0.0)))
        if not out.limit > 0 or (out.shared_ff and not out.shared_limit > 0):
            raise ValueError(f"layer {i}: the experts' limits must be positive")
        if not 0 < out.top <= out.experts + out.identity or out.experts < 1 or out.experts + out.identity > 1024:
            raise ValueError(f"layer {i}: {out.top} of {out.experts} + {out.identity} experts")
        return out

    def to_json(self) -> dict:
        out: dict = {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": []}
        for L in self.layers:
            m, f = L.mixer, L.mlp
            if isinstance(m, LatentSpec):
                kind = "latent_attention"
                mix: dict = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank,
                             "kv_rank": m.kv_rank, "scale": m.scale, "rot": {"dims": m.rot_dims, "base": m.rot_base}}
                if m.rot_scaling:
                    mix["rot"]["scaling"] = dict(m.rot_scaling)
                if m.kv_from is not None:
                    mix["kv_from"] = m.kv_from
            else:
                kind, mix = "gla", {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}
                if m.rank is not None:
                    mix["rank"] = m.rank
            mlp = None
            if f:
                mlp = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit},
                       "router": {"experts": f.experts, "identity": f.identity, "top": f.top}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff, "limit": f.shared_limit}
            out["layers"].append({"type": kind, "mixer": mix, "mlp": mlp})
        return out

    def tensor_shapes(self) -> dict[str, tuple[int | None, ...]]:
        """Every checkpoint tensor by name (None: a size that only the checkpoint knows)."""
        w = self.width
        out: dict[str, tuple[int | None, ...]] = {"embed": (self.vocab, w), "head": (self.vocab, w), "final.norm": ()}
        for i, L in enumerate(self.layers):
            m, f, p = L.mixer, L.mlp, f"l{i}."
            x = p + "mix."
            out.update({p + "norm1": (), p + "shift": (w,), p + "rg1": (w, w), p + "rg1.b": (w,)})
            if isinstance(m, LatentSpec):
                out.update({x + "dq": (m.q_rank, w), x + "dq.norm": (m.q_rank,), x + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                            x + "uk": (m.heads * m.dim, m.kv_rank), x + "uv": (m.heads * m.vdim, m.kv_rank),
                            x + "o": (w, m.heads * m.vdim)})
                if m.kv_from is None:
                    out.update({x + "dkv": (m.kv_rank + m.rot_dim, w), x + "dkv.norm": (m.kv_rank,)})
            else:
                hd, hv = m.heads * m.dim, m.heads * m.vdim
                out.update({x + "q": (hd, w), x + "k": (hd, w), x + "v": (hv, w), x + "g": (hv, w), x + "o": (w, hv), x + "norm": (m.vdim,),
                            x + "a1": (m.rank, w), x + "a2": (hd, m.rank), x + "a2.b": (hd,)})
            if f:
                y, e = p + "mlp.", f.experts + f.identity
                for j in range(f.experts):
                    out.update({f"{y}e{j}.gate": (f.ff, w), f"{y}e{j}.up": (f.ff, w), f"{y}e{j}.down": (w, f.ff)})
                out.update({y + "router": (e, w), y + "correction": (e,), p + "rg2": (w, w), p + "rg2.b": (w,)})
                if f.shared_ff:
                    out.update({y + "shared.gate": (f.shared_ff, w), y + "shared.up": (f.shared_ff, w),
                                y + "shared.down": (w, f.shared_ff), y + "shared.sg": (1, w)})
        return out

    @staticmethod
    def pattern(kinds: str, width: int, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, gla_heads: int,
                gla_dim: int, gla_vdim: int, ff: int, experts: int, identity: int, top: int, shared_ff: int, vocab: int,
                rank: int = 16) -> "KemiraxConfig":
        """Layers by letter (benchmarks, examples): ``a`` latent attention, ``b`` the same on the cache of the last ``a``,
        ``g`` gated linear attention."""
        out: list[LayerSpec] = []
        own = None
        for i, c in enumerate(kinds):
            if c == "g":
                mix: LatentSpec | LinearSpec = LinearSpec(gla_heads, gla_dim, gla_vdim, 16.0, rank)
            else:
                own = i if c == "a" else own
                mix = LatentSpec(heads, dim, rot_dim, vdim, q_rank, kv_rank, (dim + rot_dim) ** -0.5, rot_dim, 50000.0,
                                 {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}, own if c == "b" else None)
            out.append(LayerSpec(mix, ExpertsSpec(ff, 7.0, experts, identity, top, shared_ff, 7.0)))
        return KemiraxConfig(vocab, width, 1e-5, out)

    @staticmethod
    def tiny() -> "KemiraxConfig":
        return KemiraxConfig.pattern("gabg", 192, 4, 32, 16, 48, 56, 80, 3, 32, 48, 64, 6, 1, 3, 112, 512)


def synth_state(cfg: KemiraxConfig, seed: int = 0, device="cpu") -> Iterator[tuple[str, torch.Tensor]]:
    """Seeded random checkpoint tensors (bf16): projections at 1/sqrt(fan-in), norms near 1, decays spread over short and long
    memories."""
    gen = torch.Generator(device=device)
    for idx, (name, shape) in enumerate(cfg.tensor_shapes().items()):
        shape = tuple(16 if n is None else n for n in shape)
        gen.manual_seed(seed * 1_000_003 + idx)
        r = torch.randn(shape, generator=gen, device=device)
        last = name.split(".")[-1]
        if "norm" in last:
            t = 1.0 + 0.1 * r
        elif last == "shift":
            t = torch.sigmoid(r)
        elif name.endswith(".a2.b"):
            t = 2.0 + 2.0 * r
        elif name.endswith(".b"):
            t = 0.5 * r
        elif last == "correction":
            t = 0.02 * r
        elif name == "embed":
            t = r
        else:
            t = r / math.sqrt(shape[-1])
        yield name, t.bfloat16()


def write_checkpoint(directory: str, cfg: KemiraxConfig, seed: int = 0) -> None:
    """config.json + model.safetensors with random weights."""
    from ..formats import safetensors_io
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg.to_json(), f, indent=1)
    safetensors_io.write_file(os.path.join(directory, "model.safetensors"), dict(synth_state(cfg, seed)))


# ---------------------------------------------------------------------------------------------- weights
@dataclass
class LatentWeights:
    m: LatentAttention
    down: Projection                  # rows [query latent | latent | key part], or [query latent]
    uq: Projection                    # rows per head [d | r]
    uk: torch.Tensor                  # [heads, c, d]: query -> latent
    uv: torch.Tensor                  # [heads, v, c]
    ukv: Any                          # PackedLinear with rows per head [d | v]: latent -> key, value (bf16)
    o: Projection


@dataclass
class LinearWeights:
    m: GatedLinear
    proj: Projection                  # rows [q | k | v | gate | decay latent]
    o: Projection


@dataclass
class ExpertsWeights:
    spec: ExpertsSpec
    router: Projection                # rows [experts | shared expert's gate]
    correction: torch.Tensor          # fp32 [experts + identity]
    w13: moe.ExpertWeights
    w2: moe.ExpertWeights
    up: Projection | None = None      # shared expert: gate and up features interleaved in tiles (rows of the layer's ``wide``)
    down: Projection | None = None


@dataclass
class KemiraxLayer:
    mix: LatentWeights | LinearWeights
    norm: float
    shift: torch.Tensor               # fp32 [ld]
    wide: Projection                  # everything that reads the norm: rows [gates | shared expert's gate and up features]
    gates: Projection                 # its rows [mixer's gate (ld) | feed-forward's gate (ld)]
    gate_b: torch.Tensor              # fp32 [2 ld]
    ff: ExpertsWeights | None = None


def _fits(have: tuple[int, ...], want: tuple[int | None, ...]) -> bool:
    return len(have) == len(want) and all(w is None or h == w for h, w in zip(have, want))


class KemiraxWeights:
    """Device-resident, padded, kernel-ready weights from (name, tensor) pairs."""

    def __init__(self, cfg: KemiraxConfig, state, device="cuda", dtype: torch.dtype = torch.bfloat16):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("activations are bfloat16 or float32")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        t = dict(state)
        shapes = cfg.tensor_shapes()
        missing = [n for n in shapes if n not in t]
        wrong = [f"{n} {tuple(t[n].shape)} != {s}" for n, s in shapes.items() if n in t and not _fits(tuple(t[n].shape), s)]
        if missing or wrong:                       # tensors the configuration does not mention are left unread
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:4]}, shapes {wrong[:4]}")
        self.ld = pad16(cfg.width)
        self.embed = torch.zeros(cfg.vocab, self.ld, dtype=dtype, device=self.device)
        self.embed[:, :cfg.width] = t["embed"].to(self.device, dtype)
        self.head = self._proj(t["head"], pad_n=False)
        self.final_norm = float(t["final.norm"])
        self.head_lo = 0
        self.layers: list[KemiraxLayer] = []
        for i, L in enumerate(cfg.layers):
            p = f"l{i}."
            sub = lambda what: {n[len(p) + len(what) + 1:]: v for n, v in t.items() if n.startswith(p + what + ".")}
            mix = self._latent(L.mixer, sub("mix")) if isinstance(L.mixer, LatentSpec) else self._linear(L.mixer, sub("mix"))
            names = ["rg1", "rg2"] if L.mlp else ["rg1"]
            gate_b = torch.zeros(2, self.ld, dtype=torch.float32, device=self.device)
            for j, n in enumerate(names):
                gate_b[j, :cfg.width] = t[f"{p}{n}.b"].to(self.device, torch.float32)
            ff = self._experts(L.mlp, sub("mlp")) if L.mlp else None
            parts, ng = [(t[p + n], self.ld) for n in names], len(names) * self.ld
            if ff is not None and L.mlp.shared_ff:
                # rows in whole tiles of the pair GEMM, so that either part can be multiplied alone
                up = decoder.interleave_glu(t[p + "mlp.shared.gate"], t[p + "mlp.shared.up"])
                parts = [(cat_rows(parts), (ng + 255) // 256 * 256), (up, up.shape[0])]
            wide = self._proj(cat_rows(parts), tile_n=True)
            gates = wide
            if ff is not None and L.mlp.shared_ff:
                ng = parts[0][1]
                gates, ff.up = wide.part(0, ng), wide.part(ng, ng + parts[1][1])
            self.layers.append(KemiraxLayer(mix, float(t[p + "norm1"]), self._row(t[p + "shift"], self.ld), wide, gates, gate_b.view(-1), ff))

    def _proj(self, w: torch.Tensor, pad_n: bool = True, tile_n: bool = False) -> Projection:
        return Projection.make(w, self.dtype, self.device, pad_n, tile_n)

    def _row(self, w: torch.Tensor, n: int) -> torch.Tensor:
        """fp32 row padded with zeros."""
        out = torch.zeros(n, dtype=torch.float32, device=self.device)
        out[:w.numel()] = w.reshape(-1).to(self.device, torch.float32)
        return out

    def _latent(self, a: LatentSpec, t: dict[str, torch.Tensor]) -> LatentWeights:
        d, r, v, qp, c = (pad16(n) for n in (a.dim, a.rot_dim, a.vdim, a.q_rank, a.kv_rank))
        own = a.kv_from is None
        freq, mscale = yarn_freqs(a.rot_dims, a.rot_base, a.rot_scaling, self.device)
        m = LatentAttention(a.heads, a.dim, d, a.rot_dim, r, a.vdim, v, a.q_rank, qp, a.kv_rank, c, a.scale, self.cfg.eps, a.rot_dims, freq,
                            mscale, self._row(t["dq.norm"], qp), self._row(t["dkv.norm"], c) if own else None)
        parts = [(t["dq"], qp)]
        if own:
            parts += [(t["dkv"][:a.kv_rank], c), (t["dkv"][a.kv_rank:], r)]
        dev = lambda w: w.to(self.device, self.dtype).contiguous()
        uk = cat_rows([(pad_heads(t["uk"], a.heads, ((a.dim, d),)).t(), c)])                         # [c, heads * d]
        uv = torch.zeros(a.heads * v, c, dtype=t["uv"].dtype, device=t["uv"].device)
        uv[:, :a.kv_rank] = pad_heads(t["uv"], a.heads, ((a.vdim, v),))
        both = torch.cat([uk.t().reshape(a.heads, d, c), uv.view(a.heads, v, c)], 1).reshape(-1, c)
        ukv = PackedLinear.from_bf16(both.to(self.device)) if self.dtype == torch.bfloat16 else None
        return LatentWeights(m, self._proj(cat_rows(parts), tile_n=True),
                             self._proj(pad_heads(t["uq"], a.heads, ((a.dim, d), (a.rot_dim, r))), tile_n=True),
                             dev(uk.view(c, a.heads, d).permute(1, 0, 2)), dev(uv.view(a.heads, v, c)), ukv,
                             self._proj(pad_heads(t["o"].t().contiguous(), a.heads, ((a.vdim, v),)).t()))

    def _linear(self, s: LinearSpec, t: dict[str, torch.Tensor]) -> LinearWeights:
        rank = t["a1"].shape[0]
        if t["a2"].shape[1] != rank:
            raise ValueError(f"decay projection: {tuple(t['a1'].shape)} does not fit {tuple(t['a2'].shape)}")
        if s.dim > 512 or rank > 1024:
            raise ValueError("the recurrence takes up to 512 key channels per head and a decay rank of 1024")
        d, v, rp = pad16(s.dim), pad16(s.vdim), pad16(rank)
        w2 = torch.zeros(s.heads * d, rp, dtype=t["a2"].dtype, device=t["a2"].device)
        w2[:, :rank] = pad_heads(t["a2"], s.heads, ((s.dim, d),))
        m = GatedLinear(s.heads, s.dim, d, s.vdim, v, s.tau, self.cfg.eps, rp, w2.to(self.device, self.dtype).contiguous(),
                        self._row(pad_heads(t["a2.b"], s.heads, ((s.dim, d),)), s.heads * d), self._row(t["norm"], v))
        keys = [(pad_heads(t[n], s.heads, ((s.dim, d),)), s.heads * d) for n in ("q", "k")]
        values = [(pad_heads(t[n], s.heads, ((s.vdim, v),)), s.heads * v) for n in ("v", "g")]
        return LinearWeights(m, self._proj(cat_rows(keys + values + [(t["a1"], rp)]), tile_n=True),
                             self._proj(pad_heads(t["o"].t().contiguous(), s.heads, ((s.vdim, v),)).t()))

    def _experts(self, f: ExpertsSpec, t: dict[str, torch.Tensor]) -> ExpertsWeights:
        w13, w2 = moe.pack_experts(*([t[f"e{j}.{n}"] for j in range(f.experts)] for n in ("gate", "up", "down")), self.cfg.width, self.ld,
                                   self.dtype, self.device)
        rows = [(t["router"], f.experts + f.identity)] + ([(t["shared.sg"], 1)] if f.shared_ff else [])
        ew = ExpertsWeights(f, self._proj(cat_rows(rows)), self._row(t["correction"], f.experts + f.identity), w13, w2)
        if f.shared_ff:
            padded = (f.shared_ff + decoder.GLU_TILE - 1) // decoder.GLU_TILE * decoder.GLU_TILE
            down = t["shared.down"].new_zeros(self.cfg.width, padded)
            down[:, :f.shared_ff] = t["shared.down"]
            ew.down = self._proj(down)
        return ew

    def nbytes(self) -> int:
        size = lambda x: x.numel() * x.element_size()
        n = size(self.embed) + self.head.nbytes()
        for L in self.layers:
            m = L.mix
            n += L.wide.nbytes()
            n += sum(p.nbytes() for p in ((m.down, m.uq, m.o) if isinstance(m, LatentWeights) else (m.proj, m.o)))
            n += sum(size(x) for x in ((m.uk, m.uv) if isinstance(m, LatentWeights) else (m.m.w2,)))
            n += m.ukv.nbytes() if isinstance(m, LatentWeights) and m.ukv is not None else 0
            if L.ff:
                n += sum(p.nbytes() for p in (L.ff.router, L.ff.down) if p is not None)
                n += size(L.ff.w13.weight) + size(L.ff.w2.weight)
        return n


# ---------------------------------------------------------------------------------------------- runtime
class KemiraxRuntime(PagedRuntime):
    exposes_logits = True
    tile_min_rows = latent.TILE_MIN_ROWS

    def __init__(self, cfg: KemiraxConfig, weights: KemiraxWeights, max_slots: int = 1, max_context: int = 4096,
                 block_size: int = 64, num_blocks: int | None = None, comm=None):
        super().__init__(weights.device, max_slots, max_context, block_size, num_blocks, comm)
        if self.comm.world != 1:
            raise ValueError("a Kemirax model runs on one rank")
        self.cfg, self.w = cfg, weights
        tiles = weights.dtype == torch.bfloat16 and all(latent.tiles_supported(lw.mix.m) for lw in weights.layers
                                                        if isinstance(lw.mix, LatentWeights))
        if not tiles:
            self.tile_min_rows = 1 << 30             # every row on the row kernel (fp32, or heads wider than the tile kernel takes)
        self.cache: list[torch.Tensor | None] = []
        self.state: list[torch.Tensor | None] = []
        self.tails: list[torch.Tensor] = []          # the previous token's norm output, one per layer
        for i, (L, lw) in enumerate(zip(cfg.layers, weights.layers)):
            c = st = None
            if isinstance(lw.mix, LatentWeights):
                src = L.mixer.kv_from
                c = self.cache[src] if src is not None else canary.zeros(
                    self.num_blocks, block_size, lw.mix.m.cache_width, dtype=weights.dtype, device=self.device,
                    name=f"paged latent cache of layer {i}")
            else:
                m = lw.mix.m
                st = self.slot_state(m.heads, m.d, m.v, dtype=torch.float32, name=f"recurrent state of layer {i}")
            self.cache.append(c)
            self.state.append(st)
            self.tails.append(self.slot_state(weights.ld, dtype=weights.dtype, name=f"shift tail of layer {i}"))
        self.residual_tap = None                     # debugging: called with (layer, residual [T, width]) after every layer

    def _latent(self, i: int, lw: LatentWeights, y: torch.Tensor, positions, kv_slots, meta) -> torch.Tensor:
        m, cache, t = lw.m, self.cache[i], y.shape[0]
        q = lw.uq(latent.prep(lw.down(y), m, positions, kv_slots, cache))
        out = torch.empty(t, lw.o.k, dtype=y.dtype, device=y.device)
        n = meta["tile_rows"] if meta["mode"] == "mixed" else 0
        if n:                                        # portions of prompts: keys and values are expanded from the latents
            src = self.cfg.layers[i].mixer.kv_from
            src = i if src is None else src
            contexts = meta.setdefault("contexts", {})
            if src not in contexts:                  # layers that share a cache share its contiguous copy
                contexts[src] = latent.gather(cache, m, self.block_table, meta["tile_seq"], meta["kv_len"], meta["kv_start"], meta["kv_total"])
            latent.rotate_heads(q[:n], m, positions)
            latent.attend_tiles(q[:n], m, *contexts[src], lw.ukv, meta["q_start"], meta["q_len"], meta["kv_len"], meta["kv_start"],
                                meta["max_q_len"], out[:n])
        if n < t:                                    # single rows: queries are brought to the latents
            qr = q[n:]
            qa = torch.empty(t - n, m.heads, m.cache_width, dtype=y.dtype, device=y.device)
            latent.rotate_heads(qr, m, positions[n:], qa, m.c)
            latent.head_linear(qr, qr.stride(0), m.head_width, lw.uk, qa, qa.stride(0), qa.stride(1), t - n)
            if meta["mode"] == "decode":
                o = latent.attend_rows(qa, m, cache, meta["block_table"], positions, meta["max_kv_len"])
            else:
                o = latent.attend_rows(qa, m, cache, self.block_table, positions[n:], meta["max_kv_len"], seq=meta["row_seq"][n:])
            latent.head_linear(o, o.stride(0), m.c, lw.uv, out[n:], out.stride(0), m.v, t - n)
        return lw.o(out)

    def _linear(self, i: int, lw: LinearWeights, y: torch.Tensor, positions, meta) -> torch.Tensor:
        return lw.o(gla.recurrence(lw.proj(y), lw.m, self.state[i], meta["segments"], positions, lw.o.k))

    def _experts(self, ew: ExpertsWeights, h: torch.Tensor, up: torch.Tensor | None = None) -> dict:
        """``up``: the shared expert's gate and up features, where they are already there."""
        f = ew.spec
        total = f.experts + f.identity
        z = moe.router_logits(h, ew.router)
        idx, weights = moe.route(z[:, :total], ew.correction, f.top, "softmax", False, 1.0)
        y, row = moe.experts_rows(h, idx, ew.w13, ew.w2, 0, f.limit, UNIT_SLOPE)
        out = {"h": h, "routed": Routed(y, row, idx, weights, f.experts)}
        if ew.up is not None:
            unit = ew.up.glu(h, f.shared_limit, UNIT_SLOPE) if up is None else decoder.glu(up, decoder.GLU_TILE, f.shared_limit, UNIT_SLOPE)
            out.update(shared=ew.down(unit), shared_gate=z[:, total:])
        return out

    def _forward(self, ids, positions, kv_slots, meta, rows):
        cfg, w, n = self.cfg, self.w, ids.numel()
        x = torch.empty(n, w.ld, dtype=torch.float32, device=self.device)
        common = {"ld": w.ld, "n": n, "dtype": w.dtype}
        pending: dict = {"ids": ids, "table": w.embed}       # the residual starts from it

        def boundary(weight: float, **kw):
            """What is pending enters the residual; the next layer's inputs."""
            nonlocal pending
            out = decoder.parallel_step(None if "ids" in pending else x, cfg.width, weight, cfg.eps, **common, **pending, **kw)
            pending = {}
            return out

        for i, lw in enumerate(w.layers):
            h, m = boundary(lw.norm, x_out=x, shift=lw.shift, tail=self.tails[i], seg=meta["segments"], positions=positions)
            # short batches: one product for all that reads the norm; prompts: the gated unit in its GEMM's epilogue
            short = lw.ff is not None and lw.ff.up is not None and n <= SHORT_ROWS
            z = (lw.wide if short else lw.gates)(h)
            pending = {"gates": z, "gate_b": lw.gate_b}
            pending["mix"] = (self._latent(i, lw.mix, m, positions, kv_slots, meta) if isinstance(lw.mix, LatentWeights)
                              else self._linear(i, lw.mix, m, positions, meta))
            if lw.ff is not None:
                pending.update(self._experts(lw.ff, h, z[:, lw.gates.n:lw.gates.n + lw.ff.up.n] if short else None))
            if self.residual_tap is not None:
                boundary(1.0, x_out=x, norm=False)
                self.residual_tap(i, x[:, :cfg.width].clone())
        if rows is not None and rows.numel() == 0:
            return None
        return w.head(boundary(w.final_norm, rows=rows)[0], out_f32=True)


def build_synthetic(cfg: KemiraxConfig, device="cuda", seed: int = 0, dtype: torch.dtype = torch.bfloat16, **kw) -> KemiraxRuntime:
    """Random-weight runtime of the given shape."""
    return KemiraxRuntime(cfg, KemiraxWeights(cfg, synth_state(cfg, seed, device), device, dtype), **kw)
