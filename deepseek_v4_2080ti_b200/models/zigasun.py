"""Zigasun decoder: layers of differential attention (two softmax maps per head, one subtracted from the other; per-vector QK
norm, a query temperature that grows with the position, a gate per head; a layer may attend over another layer's keys and
values) and of the selective-scan mixer (Mamba), each with or without a clamped gated feed-forward.  Sublayers read the fp32
residual itself; a norm sits on their output.

The layers are described by config.json (sizes, order, constants); the passes, the pages, the state slots and the batching
come from ``models/paged.py``, the kernels from ``ops/diffattn.py``, ``ops/scan.py`` and ``ops/decoder.py``.  Activations are
bf16 (serving) or fp32 (``dtype``).
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Iterator

import torch

from ..ops import decoder, diffattn, scan
from ..ops.decoder import Projection, pad8, pad16
from ..ops.diffattn import DiffAttention
from ..utils import canary
from .paged import PagedRuntime

ARCH = "Zigasun"
# kernel sources the runtime launches (a partial build compiles only these)
KERNEL_SOURCES = ("residual_norm.cu", "bias_act.cu", "qk_head_prep.cu", "attn_diff_rows.cu", "attn_diff_prefill.cu", "conv_rows.cu",
                  "selective_scan.cu", "gemm_f32.cu", "gemm_wdec.cu", "gemm_bf16_2cta.cu", "elementwise.cu", "sampling.cu",
                  "bounds.cu")


# ---------------------------------------------------------------------------------------------- configuration
@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    temp_coef: float = 0.0
    temp_every: float = 0.0           # 0: no query temperature
    kv_from: int | None = None        # attends over this layer's keys and values


@dataclass
class ScanSpec:
    inner: int
    state: int
    dt_rank: int
    conv: int                         # taps


@dataclass
class LayerSpec:
    mixer: AttentionSpec | ScanSpec
    ff: int = 0                       # 0: no feed-forward
    limit: float = 0.0


@dataclass
class ZigasunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    layers: list[LayerSpec] = field(default_factory=list)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def is_zigasun_json(raw: Any) -> bool:
        return isinstance(raw, dict) and raw.get("architecture") == ARCH

    @staticmethod
    def from_json(raw: dict) -> "ZigasunConfig":
        if not ZigasunConfig.is_zigasun_json(raw):
            raise ValueError(f"not a {ARCH} configuration")
        layers: list[LayerSpec] = []
        for i, L in enumerate(raw["layers"]):
            m, mlp = L["mixer"], L.get("mlp")
            if L["type"] == "attention":
                temp = m.get("q_temp") or {}
                src = m.get("kv_from")
                mix: AttentionSpec | ScanSpec = AttentionSpec(
                    int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), float(m["scale"]),
                    float(m["diff"]), float(temp.get("coef", 0.0)), float(temp.get("every", 0.0)), None if src is None else int(src))
                if mix.heads % mix.kv_heads:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if src is not None:
                    o = layers[mix.kv_from].mixer if 0 <= mix.kv_from < i else None
                    if not isinstance(o, AttentionSpec) or o.kv_from is not None or \
                            (o.kv_heads, o.dim, o.vdim) != (mix.kv_heads, mix.dim, mix.vdim):
                        raise ValueError(f"layer {i}: kv_from {src} is not an earlier attention layer with equal key/value heads of its own")
            elif L["type"] == "mamba1":
                mix = ScanSpec(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
            else:
                raise ValueError(f"layer {i}: mixer type {L['type']!r} is not one of this design")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not one of this design")
            if mlp and not float(mlp["limit"]) > 0:
                raise ValueError(f"layer {i}: the feed-forward's limit must be positive")
            layers.append(LayerSpec(mix, int(mlp["ff"]) if mlp else 0, float(mlp["limit"]) if mlp else 0.0))
        return ZigasunConfig(int(raw["vocab"]), int(raw["width"]), float(raw["norm"]["eps"]),
                             float((raw.get("embedding") or {}).get("scale", 1.0)), float(raw.get("residual_mult", 1.0)), layers)

    def to_json(self) -> dict:
        out: dict = {"architecture": ARCH, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                     "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult, "layers": []}
        for L in self.layers:
            m = L.mixer
            if isinstance(m, AttentionSpec):
                kind = "attention"
                mix: dict = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "diff": m.diff}
                if m.temp_every:
                    mix["q_temp"] = {"coef": m.temp_coef, "every": m.temp_every}
                if m.kv_from is not None:
                    mix["kv_from"] = m.kv_from
            else:
                kind, mix = "mamba1", {"inner": m.inner, "state": m.state, "dt_rank": m.dt_rank, "conv": m.conv}
            out["layers"].append({"type": kind, "mixer": mix, "mlp": {"kind": "dense", "ff": L.ff, "limit": L.limit} if L.ff else None})
        return out

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every checkpoint tensor by name."""
        w = self.width
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab, w), "head": (self.vocab, w), "final.norm": (w,)}
        for i, L in enumerate(self.layers):
            m, p = L.mixer, f"l{i}."
            x = p + "mix."
            out[p + "norm1"] = (w,)
            if isinstance(m, AttentionSpec):
                out.update({x + "q": (m.heads * 2 * m.dim, w), x + "q.norm": (m.dim,), x + "g": (m.heads, w), x + "o": (w, m.heads * m.vdim)})
                out.update({x + n: (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
                if m.kv_from is None:
                    out.update({x + "k": (m.kv_heads * 2 * m.dim, w), x + "v": (m.kv_heads * m.vdim, w), x + "k.norm": (m.dim,)})
            else:
                out.update({x + "in": (2 * m.inner, w), x + "conv": (m.inner, m.conv), x + "conv.b": (m.inner,),
                            x + "x": (m.dt_rank + 2 * m.state, m.inner), x + "dt": (m.inner, m.dt_rank), x + "dt.b": (m.inner,),
                            x + "A_log": (m.inner, m.state), x + "D": (m.inner,), x + "o": (w, m.inner)})
            if L.ff:
                out.update({p + "norm2": (w,), p + "mlp.gate": (L.ff, w), p + "mlp.up": (L.ff, w), p + "mlp.down": (w, L.ff)})
        return out

    @staticmethod
    def alternating(layers: int, width: int, heads: int, kv_heads: int, dim: int, vdim: int, ff: int, inner: int, state: int,
                    dt_rank: int, vocab: int, share: bool = False) -> "ZigasunConfig":
        """Attention with a feed-forward and a scan layer in turn (benchmarks, examples); ``share``: attention layers after
        the first use its keys and values."""
        out = []
        for i in range(layers):
            if i % 2 == 0:
                out.append(LayerSpec(AttentionSpec(heads, kv_heads, dim, vdim, dim ** -0.5, 0.2, 0.1, 4096,
                                                   0 if share and i else None), ff, 7.0))
            else:
                out.append(LayerSpec(ScanSpec(inner, state, dt_rank, 4)))
        return ZigasunConfig(vocab, width, 1e-5, 1.0, 1.0, out)

    @staticmethod
    def tiny() -> "ZigasunConfig":
        return ZigasunConfig.alternating(5, 192, 6, 3, 32, 64, 384, 256, 16, 12, 512, share=True)


def synth_state(cfg: ZigasunConfig, seed: int = 0, device="cpu") -> Iterator[tuple[str, torch.Tensor]]:
    """Seeded random checkpoint tensors (bf16): projections at 1/sqrt(fan-in), norms near 1, decays and step sizes spread
    over short and long memories."""
    gen = torch.Generator(device=device)
    for idx, (name, shape) in enumerate(cfg.tensor_shapes().items()):
        gen.manual_seed(seed * 1_000_003 + idx)
        r = torch.randn(shape, generator=gen, device=device)
        last = name.split(".")[-1]
        if "norm" in last:
            t = 1.0 + 0.1 * r
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.5 * r / math.sqrt(math.sqrt(shape[0]))
        elif name.endswith(".A_log"):
            t = torch.log(torch.arange(1, shape[1] + 1, device=device, dtype=torch.float32)).expand(shape) + 0.1 * r
        elif name.endswith(".dt.b"):
            t = -3.0 + 1.5 * r
        elif name.endswith(".conv"):
            t = r / math.sqrt(shape[1])
        elif name.endswith(".conv.b"):
            t = 0.2 * r
        elif name.endswith(".D"):
            t = 1.0 + 0.2 * r
        elif name == "embed":
            t = r
        else:
            t = r / math.sqrt(shape[-1])
        yield name, t.bfloat16()


def write_checkpoint(directory: str, cfg: ZigasunConfig, seed: int = 0) -> None:
    """config.json + model.safetensors with random weights."""
    from ..formats import safetensors_io
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg.to_json(), f, indent=1)
    safetensors_io.write_file(os.path.join(directory, "model.safetensors"), dict(synth_state(cfg, seed)))


# ---------------------------------------------------------------------------------------------- weights
@dataclass
class AttentionWeights:
    m: DiffAttention
    proj: Projection                  # rows [queries | keys | values | gates], or [queries | gates]
    gate_off: int
    o: Projection


@dataclass
class ScanWeights:
    inner: int                        # padded channels
    in_: Projection                   # rows [x | z]
    conv: torch.Tensor                # fp32 [taps, inner]
    conv_b: torch.Tensor
    x: Projection                     # rows [dt rank | B | C], each part padded to a multiple of 8
    b_off: int
    c_off: int
    dt: Projection                    # zero columns for the B and C parts, so that it reads the whole row
    dt_b: torch.Tensor
    a: torch.Tensor
    d: torch.Tensor
    o: Projection


@dataclass
class ZigasunLayer:
    mix: AttentionWeights | ScanWeights
    norm1: torch.Tensor               # with the residual multiplier in it
    norm2: torch.Tensor | None = None
    up: Projection | None = None      # gate and up features interleaved in tiles
    down: Projection | None = None
    limit: float = 0.0


class ZigasunWeights:
    """Device-resident, padded, kernel-ready weights from (name, tensor) pairs."""

    def __init__(self, cfg: ZigasunConfig, state, device="cuda", dtype: torch.dtype = torch.bfloat16):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("activations are bfloat16 or float32")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        t = dict(state)
        shapes = cfg.tensor_shapes()
        missing = [n for n in shapes if n not in t]
        wrong = [f"{n} {tuple(t[n].shape)} != {s}" for n, s in shapes.items() if n in t and tuple(t[n].shape) != s]
        if missing or wrong:                       # tensors the configuration does not mention are left unread
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:4]}, shapes {wrong[:4]}")
        self.ld = pad16(cfg.width)
        self.embed = torch.zeros(cfg.vocab, self.ld, dtype=dtype, device=self.device)
        self.embed[:, :cfg.width] = t["embed"].to(self.device, dtype)
        self.head = self._proj(t["head"], pad_n=False)
        self.final_norm = self._row(t["final.norm"])
        self.head_lo = 0
        self.layers: list[ZigasunLayer] = []
        for i, L in enumerate(cfg.layers):
            p = f"l{i}."
            sub = {n[len(p) + 4:]: v for n, v in t.items() if n.startswith(p + "mix.")}
            mix = self._attention(L.mixer, sub) if isinstance(L.mixer, AttentionSpec) else self._scan(L.mixer, sub)
            lw = ZigasunLayer(mix, self._row(t[p + "norm1"], scale=cfg.residual_mult))
            if L.ff:
                lw.norm2 = self._row(t[p + "norm2"], scale=cfg.residual_mult)
                lw.up = self._proj(decoder.interleave_glu(t[p + "mlp.gate"], t[p + "mlp.up"]))
                down = torch.zeros(cfg.width, lw.up.n // 2, dtype=t[p + "mlp.down"].dtype, device=t[p + "mlp.down"].device)
                down[:, :L.ff] = t[p + "mlp.down"]
                lw.down, lw.limit = self._proj(down), L.limit
            self.layers.append(lw)

    def _proj(self, w: torch.Tensor, pad_n: bool = True, tile_n: bool = False) -> Projection:
        return Projection.make(w, self.dtype, self.device, pad_n, tile_n)

    def _row(self, w: torch.Tensor, n: int | None = None, scale: float = 1.0) -> torch.Tensor:
        """fp32 row padded with zeros to n (default: the residual's width)."""
        out = torch.zeros(n or self.ld, dtype=torch.float32, device=self.device)
        out[:w.numel()] = w.to(self.device, torch.float32) * scale
        return out

    def _attention(self, a: AttentionSpec, t: dict[str, torch.Tensor]) -> AttentionWeights:
        d, v = pad16(a.dim), pad16(a.vdim)

        def vectors(w: torch.Tensor, n: int, real: int, padded: int) -> torch.Tensor:
            """[n * real, ...] -> [n * padded, ...]: zero rows after every vector."""
            out = torch.zeros(n, padded, *w.shape[1:], dtype=w.dtype, device=w.device)
            out[:, :real] = w.reshape(n, real, *w.shape[1:])
            return out.reshape(n * padded, *w.shape[1:])

        f64 = {n: t[n].double() for n in ("lq1", "lk1", "lq2", "lk2")}
        lam = float(torch.exp((f64["lq1"] * f64["lk1"]).sum()) - torch.exp((f64["lq2"] * f64["lk2"]).sum())) + a.diff
        own = a.kv_from is None
        m = DiffAttention(a.heads, a.kv_heads, a.dim, d, a.vdim, v, a.scale, lam, a.diff, self.cfg.eps, self._row(t["q.norm"], d),
                          self._row(t["k.norm"], d) if own else None, a.temp_coef, a.temp_every)
        parts = [vectors(t["q"], 2 * a.heads, a.dim, d)]
        if own:
            parts += [vectors(t["k"], 2 * a.kv_heads, a.dim, d), vectors(t["v"], a.kv_heads, a.vdim, v)]
        gate_off = sum(w.shape[0] for w in parts)
        o = vectors(t["o"].t().contiguous(), a.heads, a.vdim, v).t()
        return AttentionWeights(m, self._proj(torch.cat(parts + [t["g"]]), tile_n=True), gate_off, self._proj(o))

    def _scan(self, s: ScanSpec, t: dict[str, torch.Tensor]) -> ScanWeights:
        if not 0 < s.state <= 256:
            raise ValueError("the scan kernel takes up to 256 states per channel")
        ip, r8, n8 = pad16(s.inner), pad8(s.dt_rank), pad8(s.state)
        wi = torch.zeros(2, ip, self.cfg.width, dtype=t["in"].dtype, device=t["in"].device)
        wi[:, :s.inner] = t["in"].view(2, s.inner, -1)
        wx = torch.zeros(pad16(r8 + 2 * n8), ip, dtype=t["x"].dtype, device=t["x"].device)
        for lo, at, n in ((0, 0, s.dt_rank), (s.dt_rank, r8, s.state), (s.dt_rank + s.state, r8 + n8, s.state)):
            wx[at:at + n, :s.inner] = t["x"][lo:lo + n]
        wd = torch.zeros(ip, wx.shape[0], dtype=t["dt"].dtype, device=t["dt"].device)
        wd[:s.inner, :s.dt_rank] = t["dt"]
        conv = torch.zeros(s.conv, ip, dtype=torch.float32, device=self.device)
        conv[:, :s.inner] = t["conv"].to(self.device, torch.float32).t()
        a = torch.zeros(ip, s.state, dtype=torch.float32, device=self.device)
        a[:s.inner] = scan.scan_decay(t["A_log"].to(self.device), self.dtype)
        return ScanWeights(ip, self._proj(wi.view(2 * ip, -1)), conv, self._row(t["conv.b"], ip), self._proj(wx), r8, r8 + n8,
                           self._proj(wd), self._row(t["dt.b"], ip), a, self._row(t["D"], ip), self._proj(t["o"]))

    def nbytes(self) -> int:
        n = self.embed.numel() * self.embed.element_size() + self.head.nbytes()
        for L in self.layers:
            m = L.mix
            own = (m.proj, m.o) if isinstance(m, AttentionWeights) else (m.in_, m.x, m.dt, m.o)
            n += sum(p.nbytes() for p in (*own, L.up, L.down) if p is not None)
        return n


# ---------------------------------------------------------------------------------------------- runtime
class ZigasunRuntime(PagedRuntime):
    exposes_logits = True
    tile_min_rows = diffattn.TILE_MIN_ROWS

    def __init__(self, cfg: ZigasunConfig, weights: ZigasunWeights, max_slots: int = 1, max_context: int = 4096,
                 block_size: int = 64, num_blocks: int | None = None, comm=None):
        super().__init__(weights.device, max_slots, max_context, block_size, num_blocks, comm)
        if self.comm.world != 1:
            raise ValueError("a Zigasun model runs on one rank")
        self.cfg, self.w = cfg, weights
        self.k_cache: list[torch.Tensor | None] = []
        self.v_cache: list[torch.Tensor | None] = []
        self.conv_tail: list[torch.Tensor | None] = []
        self.scan_state: list[torch.Tensor | None] = []
        pages = lambda width, what: canary.zeros(self.num_blocks, block_size, width, dtype=weights.dtype, device=self.device, name=what)
        tiles = weights.dtype == torch.bfloat16
        for i, (L, lw) in enumerate(zip(cfg.layers, weights.layers)):
            k = v = tail = st = None
            if isinstance(lw.mix, AttentionWeights):
                m, src = lw.mix.m, L.mixer.kv_from
                if src is not None:
                    k, v = self.k_cache[src], self.v_cache[src]
                else:
                    k, v = pages(m.k_width, f"paged key cache of layer {i}"), pages(m.v_width, f"paged value cache of layer {i}")
                tiles = tiles and diffattn.tiles_supported(m, block_size)
            else:
                s = L.mixer
                tail = self.slot_state(max(s.conv - 1, 1), lw.mix.inner, dtype=weights.dtype, name=f"convolution tail of layer {i}")
                st = self.slot_state(lw.mix.inner, s.state, dtype=torch.float32, name=f"scan state of layer {i}")
            self.k_cache.append(k)
            self.v_cache.append(v)
            self.conv_tail.append(tail)
            self.scan_state.append(st)
        if not tiles:
            self.tile_min_rows = 1 << 30          # every row on the row kernel (fp32, or vectors wider than the tile kernel takes)
        self.residual_tap = None                  # debugging: called with (layer, residual [T, width]) after every layer

    def _attention(self, i: int, aw: AttentionWeights, y: torch.Tensor, positions, kv_slots, meta) -> torch.Tensor:
        m, k, v = aw.m, self.k_cache[i], self.v_cache[i]
        t = y.shape[0]
        n = meta["tile_rows"] if meta["mode"] == "mixed" else 0
        proj = aw.proj(y)
        gate = proj[:, aw.gate_off:]
        q = diffattn.head_prep(proj, m, positions, kv_slots, k, v)
        out = torch.empty(t, aw.o.k, dtype=y.dtype, device=y.device)
        if n:
            diffattn.prefill(q[:n], m, k, v, gate, self.block_table, meta["q_start"], meta["q_len"], meta["kv_len"],
                             meta["max_q_len"], out[:n], seq=meta["tile_seq"])
        if n < t:
            if meta["mode"] == "decode":
                diffattn.rows(q, m, k, v, gate, meta["block_table"], positions, meta["max_kv_len"], out)
            else:
                diffattn.rows(q[n:], m, k, v, gate[n:], self.block_table, positions[n:], meta["max_kv_len"], out[n:],
                              seq=meta["row_seq"][n:])
        return aw.o(out)

    def _scan(self, i: int, sw: ScanWeights, y: torch.Tensor, positions, meta) -> torch.Tensor:
        seg, tail = meta["segments"], self.conv_tail[i]
        xz = sw.in_(y)
        x_in, z = xz[:, :sw.inner], xz[:, sw.inner:]
        x = scan.conv_rows(x_in, sw.conv, sw.conv_b, tail, seg, positions)
        p = sw.x(x)
        dt = sw.dt(p, out_f32=True)
        return sw.o(scan.selective_scan(x, dt, p, sw.b_off, sw.c_off, z, sw.a, sw.dt_b, sw.d, self.scan_state[i], seg, positions,
                                        x_in, tail))

    def _forward(self, ids, positions, kv_slots, meta, rows):
        cfg, w = self.cfg, self.w
        x = torch.empty(ids.numel(), w.ld, dtype=torch.float32, device=self.device)
        exact = w.dtype == torch.float32
        pending: dict = {"ids": ids, "table": w.embed, "table_scale": cfg.embedding_scale}      # the residual starts from it

        def boundary(**kw):
            """What is pending enters the residual; the next sublayer's input (the residual itself in fp32)."""
            nonlocal pending
            out = decoder.residual_norm(x, cfg.width, cfg.eps, dtype=w.dtype, rms=True, **pending, **kw)
            pending = {}
            return x if exact and "pre_w" not in kw else out

        for i, lw in enumerate(w.layers):
            y = boundary(plain=not exact)
            out = (self._attention(i, lw.mix, y, positions, kv_slots, meta) if isinstance(lw.mix, AttentionWeights)
                   else self._scan(i, lw.mix, y, positions, meta))
            pending = {"delta": out, "post_w": lw.norm1}
            if lw.up is not None:
                y = boundary(plain=not exact)
                pending = {"delta": lw.down(lw.up.glu(y, lw.limit)), "post_w": lw.norm2}
            if self.residual_tap is not None:
                boundary()
                self.residual_tap(i, x[:, :cfg.width].clone())
        if rows is not None and rows.numel() == 0:
            return None
        return w.head(boundary(pre_w=w.final_norm, rows=rows), out_f32=True)


def build_synthetic(cfg: ZigasunConfig, device="cuda", seed: int = 0, dtype: torch.dtype = torch.bfloat16, **kw) -> ZigasunRuntime:
    """Random-weight runtime of the given shape."""
    return ZigasunRuntime(cfg, ZigasunWeights(cfg, synth_state(cfg, seed, device), device, dtype), **kw)
