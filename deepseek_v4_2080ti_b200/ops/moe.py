"""Routed-expert MoE on the GPU: router top-k, device-side planning, grouped tcgen05 GEMMs over expert-sorted rows
(csrc/kernels/moe.cu + the grouped mode of csrc/kernels/gemm_wdec.cu).  No host synchronisation anywhere: the
number of rows per expert only exists on the device."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib, gemm
from .gemm import WF_BF16, WF_FP8_B128

WF_FP4 = 2
WF_F32 = 100                   # not a GEMM format: plain fp32 matrices on the CUDA cores (gemm_f32.cu)
# softmax_chosen: softmax over the chosen logits only, the bias belongs to the logits
SCORE_FN = {"softmax": 0, "sigmoid": 1, "sqrtsoftplus": 2, "softmax_chosen": 3}


def prepack_fp4(packed: torch.Tensor, scale_e8m0: torch.Tensor) -> torch.Tensor:
    """FP4 weight (uint8 [N, K/2] two codes per byte, low nibble first; E8M0 uint8 [N, K/32]) -> the GEMM's
    tile-major layout uint8 [ceil(N/128), K/64, 4352]: per stage 128 rows x 32 code bytes, then 128 x 2 scale bytes."""
    n, kh = packed.shape
    k = kh * 2
    assert k % 64 == 0 and scale_e8m0.shape == (n, k // 32)
    npad = (n + 127) // 128 * 128
    if npad != n:
        packed = torch.cat([packed, packed.new_zeros(npad - n, kh)])
        scale_e8m0 = torch.cat([scale_e8m0, scale_e8m0.new_zeros(npad - n, k // 32)])
    codes = packed.view(npad // 128, 128, k // 64, 32).permute(0, 2, 1, 3).reshape(npad // 128, k // 64, 128 * 32)
    sc = scale_e8m0.view(npad // 128, 128, k // 64, 2).permute(0, 2, 1, 3).reshape(npad // 128, k // 64, 128 * 2)
    return torch.cat([codes, sc], -1).contiguous()


@dataclass
class ExpertWeights:
    """Stacked weights of this rank's experts for one grouped GEMM."""
    wfmt: int
    weight: torch.Tensor            # fp4/fp8: uint8 [E, mt, kb, stage_bytes]; bf16: [E*N, K]
    scales: torch.Tensor | None     # fp8: fp32 [E, ceil(N/128), K/128]
    n: int
    k: int
    experts: int

    @staticmethod
    def from_fp4(packed: list[torch.Tensor], scales: list[torch.Tensor]) -> "ExpertWeights":
        n, kh = packed[0].shape
        w = torch.stack([prepack_fp4(p, s) for p, s in zip(packed, scales)])
        return ExpertWeights(WF_FP4, w, None, n, kh * 2, len(packed))

    @staticmethod
    def from_fp8(ws: list[torch.Tensor], scales: list[torch.Tensor]) -> "ExpertWeights":
        n, k = ws[0].shape
        w = torch.stack([gemm.prepack_fp8(x) for x in ws])
        return ExpertWeights(WF_FP8_B128, w, torch.stack([s.float() for s in scales]).contiguous(), n, k, len(ws))

    @staticmethod
    def from_gguf(raws: list[torch.Tensor], ggml_type, n: int, k: int) -> "ExpertWeights":
        """Raw GGUF blocks (uint8 [N, row_bytes]) of each expert -> stage-major stacks decoded inside the grouped GEMM.
        ``scales`` carries the codebook table for the formats that need one."""
        from . import gguf_gemm
        w = torch.stack([gguf_gemm.prepack(r, ggml_type, k) for r in raws])
        lut = gguf_gemm.lut_for(ggml_type, raws[0].device)
        return ExpertWeights(gguf_gemm.WF[gguf_gemm.GGMLType(ggml_type)], w, lut, n, k, len(raws))

    @staticmethod
    def from_f32(ws: list[torch.Tensor]) -> "ExpertWeights":
        n, k = ws[0].shape
        return ExpertWeights(WF_F32, torch.cat([x.float() for x in ws]).contiguous(), None, n, k, len(ws))

    @staticmethod
    def from_bf16(ws: list[torch.Tensor]) -> "ExpertWeights":
        n, k = ws[0].shape
        assert n % 128 == 0, "bf16 expert matrices need a multiple of 128 output features"
        return ExpertWeights(WF_BF16, torch.cat([x.to(torch.bfloat16) for x in ws]).contiguous(), None, n, k, len(ws))


ROUTER_MAX_ROWS = 64            # batches up to this take the row kernel: a tensor-core tile would leave all but one SM idle


def router_logits(x: torch.Tensor, w) -> torch.Tensor:
    """fp32 logits [T, w.n] of a router (``ops.decoder.Projection``)."""
    if x.dtype != torch.bfloat16 or x.shape[0] > ROUTER_MAX_ROWS:
        return w(x, out_f32=True)
    t, k = x.shape
    assert x.is_contiguous() and k == w.k
    z = torch.empty(t, w.n, dtype=torch.float32, device=x.device)
    rc = _lib.lib().b200_rows_linear_f32(_lib.ptr(x), k, _lib.ptr(w.packed.weight), _lib.ptr(z), w.n, t, w.n, k, _lib.stream())
    _lib.check(rc, "rows_linear")
    return z


def route(logits: torch.Tensor, bias: torch.Tensor | None, k: int, score_func: str, norm_topk: bool,
          route_scale: float) -> tuple[torch.Tensor, torch.Tensor]:
    """fp32 logits [T, E] (row stride allowed) -> (idx int32 [T, k], weights fp32 [T, k])."""
    t, e = logits.shape
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    idx = torch.empty(t, k, dtype=torch.int32, device=logits.device)
    wts = torch.empty(t, k, dtype=torch.float32, device=logits.device)
    rc = _lib.lib().b200_moe_route(_lib.ptr(logits), logits.stride(0), _lib.ptr(bias), t, e, k, SCORE_FN[score_func],
                                   int(norm_topk), ctypes.c_float(route_scale), _lib.ptr(idx), _lib.ptr(wts), _lib.stream())
    _lib.check(rc, "moe_route")
    return idx, wts


def pack_experts(gate: list[torch.Tensor], up: list[torch.Tensor], down: list[torch.Tensor], width: int, ld: int, dtype: torch.dtype,
                 device) -> tuple[ExpertWeights, ExpertWeights]:
    """Gate, up [ff, width] and down [width, ff] of every expert, padded for the grouped GEMM on rows of ``ld`` columns."""
    f32, real = dtype == torch.float32, gate[0].shape[0]
    ff = (real + 15) // 16 * 16 if f32 else (real + 63) // 64 * 64     # the grouped GEMM tiles features by 128, gate and up together
    out = ld if f32 else (ld + 127) // 128 * 128
    w13, w2 = [], []
    for g, u, d in zip(gate, up, down):
        a = torch.zeros(2, ff, ld, dtype=dtype, device=device)
        a[0, :real, :width] = g.to(device, dtype)
        a[1, :real, :width] = u.to(device, dtype)
        b = torch.zeros(out, ff, dtype=dtype, device=device)
        b[:width, :real] = d.to(device, dtype)
        w13.append(a.view(2 * ff, ld))
        w2.append(b)
    pack = ExpertWeights.from_f32 if f32 else ExpertWeights.from_bf16
    return pack(w13), pack(w2)


F32_TILE = 64                   # rows and features of a tile of the fp32 grouped GEMM


def experts_rows(x: torch.Tensor, idx: torch.Tensor, w13: ExpertWeights, w2: ExpertWeights, expert_lo: int = 0,
                 limit: float = 0.0, slope: float = 0.0) -> tuple[torch.Tensor, torch.Tensor]:
    """Outputs of the experts [expert_lo, expert_lo + E) held here for their tokens, in expert order (y [T k, w2.n]), and the
    row of every route (int32 [T, k], -1: not held here).  x [T, H] bf16 (fp32 for fp32 weights); w13: [E] x [2I, H] (gate
    rows then up rows); w2: [E] x [H', I].  The unit is SwiGLU with the optional clamp ``limit``, or with ``slope`` the
    clamped one-plus form of csrc/kernels/glu.cuh."""
    L = _lib.lib()
    t, h = x.shape
    k = idx.shape[1]
    el = w13.experts
    inter = w13.n // 2
    r = t * k
    dev = x.device
    f32 = w13.wfmt == WF_F32
    assert x.dtype == (torch.float32 if f32 else torch.bfloat16) and x.is_contiguous() and h == w13.k
    bn = F32_TILE if f32 else gemm._bn(min(256, max(16, (r + el - 1) // el)))      # token tile sized for the average rows per expert
    if 3 <= w13.wfmt < WF_F32:
        bn = min(bn, int(L.b200_gguf_max_bn(w13.wfmt)), int(L.b200_gguf_max_bn(w2.wfmt)))
    bm = F32_TILE if f32 else 128
    mt13, mt2 = (w13.n + bm - 1) // bm, (w2.n + bm - 1) // bm
    max_work = (mt13 + mt2) * ((r + bn - 1) // bn + el)
    i32 = lambda *s: torch.empty(*s, dtype=torch.int32, device=dev)
    offsets, route_row, row_token = i32(el + 1), i32(t, k), i32(r)
    work13, work2 = i32(max_work, 4), i32(max_work, 4)
    n13, n2 = i32(1), i32(1)
    s = _lib.stream()
    rc = L.b200_moe_plan(_lib.ptr(idx), t, k, expert_lo, expert_lo + el, _lib.ptr(offsets), _lib.ptr(route_row),
                         _lib.ptr(row_token), _lib.ptr(work13), _lib.ptr(n13), mt13, bn, _lib.ptr(work2), _lib.ptr(n2),
                         mt2, bn, max_work, s)
    _lib.check(rc, "moe_plan")
    # rows past the real count are never read: sized for the worst case (every route local)
    xs = torch.empty(r, h, dtype=x.dtype, device=dev)
    # 16-bit columns: an fp32 row counts twice
    rc = L.b200_moe_gather(_lib.ptr(x), _lib.ptr(row_token), _lib.ptr(offsets), el, _lib.ptr(xs), r, 2 * h if f32 else h, s)
    _lib.check(rc, "moe_gather")

    def product(w: ExpertWeights, a: torch.Tensor, work, num, what: str) -> torch.Tensor:
        out = torch.empty(r, w.n, dtype=x.dtype, device=dev)
        if f32:
            rc = L.b200_gemm_f32_grouped(_lib.ptr(a), _lib.ptr(w.weight), _lib.ptr(out), w.n, w.k, _lib.ptr(work), _lib.ptr(num),
                                         max_work, s)
        else:
            grouped = L.b200_gemm_wdec_grouped if w.wfmt < 3 else L.b200_gemm_wdec_gguf_grouped
            rc = grouped(w.wfmt, _lib.ptr(w.weight), _lib.ptr(w.scales), _lib.ptr(a), _lib.ptr(out), r, w.n, w.k, el,
                         _lib.ptr(work), _lib.ptr(num), bn, _lib.ptr(_lib.status_word(dev)), s)
        _lib.check(rc, what)
        return out

    gu = product(w13, xs, work13, n13, "grouped gemm w13")
    act = torch.empty(r, inter, dtype=x.dtype, device=dev)
    rc = L.b200_moe_glu(_lib.ptr(gu), _lib.ptr(offsets), el, _lib.ptr(act), r, inter, ctypes.c_float(limit), ctypes.c_float(slope),
                        int(f32), s)
    _lib.check(rc, "moe_glu")
    return product(w2, act, work2, n2, "grouped gemm w2"), route_row


def experts_forward(x: torch.Tensor, idx: torch.Tensor, wts: torch.Tensor, w13: ExpertWeights, w2: ExpertWeights,
                    expert_lo: int, swiglu_limit: float = 0.0, base: torch.Tensor | None = None, comm=None,
                    residual: torch.Tensor | None = None, comm_mode: int = 0) -> torch.Tensor:
    """out[t] = base[t] + sum_k wts[t,k] * Expert_{idx[t,k]}(x[t]) over the experts [expert_lo, expert_lo + E) held here.
    x [T, H] bf16; w13: [E] x [2I, H] (gate rows then up rows); w2: [E] x [H, I].

    With ``comm`` (a peer-memory communicator of an expert-parallel group) the weighted combine, the sum over ranks
    and the residual add run as one kernel over NVLink (``PeerComm.moe_combine``): every rank gets
    ``residual + sum_ranks(base_r + local routes)``."""
    t, h = x.shape
    k = idx.shape[1]
    y, route_row = experts_rows(x, idx, w13, w2, expert_lo, swiglu_limit)
    if comm is not None and getattr(comm, "world", 1) > 1:
        return comm.moe_combine(y, route_row, wts, base, residual, t, k, h, comm_mode)
    if residual is not None:
        base = residual if base is None else base + residual
    out = torch.empty(t, h, dtype=torch.bfloat16, device=x.device)
    rc = _lib.lib().b200_moe_combine(_lib.ptr(y), _lib.ptr(route_row), _lib.ptr(wts), _lib.ptr(base), _lib.ptr(out), t, k, h,
                                     _lib.stream())
    _lib.check(rc, "moe_combine")
    return out


class OffloadedExperts:
    """Routed experts of one layer kept in pinned host memory with ``capacity`` device slots per matrix
    (``components.expert_cache.HotExpertCache``): a call copies in the experts its tokens route to (least recently
    used ones make room), rewrites the routing ids to slot numbers and runs the ordinary grouped GEMMs over the slot
    arrays.  For models whose experts do not fit beside the caches, and for prefill, where a chunk touches most
    experts once and the copies overlap the previous layer.  A chunk that routes to more experts than there are slots
    is split in halves by tokens.  Reference: GPUPrefillMoEBackend with its hot-expert cache
    (src/components/moe/gpu_prefill_backend.py:41-104, 105-901)."""

    def __init__(self, w13: ExpertWeights, w2: ExpertWeights, capacity: int, device, expert_lo: int = 0):
        from ..components.expert_cache import HotExpertCache
        assert w13.experts == w2.experts and (w13.scales is None or w13.wfmt >= 3) and (w2.scales is None or w2.wfmt >= 3), \
            "per-expert scale grids (FP8) are not packed into the slabs"
        self.experts, self.expert_lo = w13.experts, int(expert_lo)
        self.capacity = min(int(capacity), self.experts)
        self.dev = torch.device(device)

        def split(w: ExpertWeights):
            per = w.weight.reshape(w.experts, -1)
            host = per.contiguous().view(torch.uint8).cpu()
            cache = HotExpertCache(host, self.capacity, self.dev)
            shape = (self.capacity * w.n, w.k) if w.wfmt == WF_BF16 else (self.capacity, *w.weight.shape[1:])
            view = cache.slots.view(w.weight.dtype).view(*shape)
            lut = w.scales.to(self.dev) if w.scales is not None else None
            return cache, ExpertWeights(w.wfmt, view, lut, w.n, w.k, self.capacity)

        self.c13, self.w13 = split(w13)
        self.c2, self.w2 = split(w2)

    def stats(self) -> dict:
        a, b = self.c13.stats, self.c2.stats
        return {"hits": a.hits + b.hits, "misses": a.misses + b.misses, "evictions": a.evictions + b.evictions,
                "bytes_copied": a.bytes_copied + b.bytes_copied}

    def forward(self, x: torch.Tensor, idx: torch.Tensor, wts: torch.Tensor, swiglu_limit: float = 0.0,
                base: torch.Tensor | None = None) -> torch.Tensor:
        lo, hi = self.expert_lo, self.expert_lo + self.experts
        local = (idx >= lo) & (idx < hi)
        need = torch.unique(idx[local]).tolist()                       # host sync: the copies depend on the routing
        if len(need) > self.capacity and x.shape[0] > 1:
            h = x.shape[0] // 2
            parts = [self.forward(x[a:b].contiguous(), idx[a:b].contiguous(), wts[a:b].contiguous(), swiglu_limit,
                                  None if base is None else base[a:b].contiguous()) for a, b in ((0, h), (h, x.shape[0]))]
            return torch.cat(parts)
        if len(need) > self.capacity:
            raise RuntimeError(f"one token routes to {len(need)} experts of this rank; the cache holds {self.capacity}")
        local_ids = [e - lo for e in need]
        s13, s2 = self.c13.fetch(local_ids), self.c2.fetch(local_ids)
        assert torch.equal(s13, s2), "the two caches see the same requests and must agree on the slots"
        table = torch.full((self.experts + 1,), self.capacity, dtype=torch.int32, device=idx.device)
        if local_ids:
            table[torch.tensor(local_ids, dtype=torch.long, device=idx.device)] = s13.to(idx.device)
        # ids of other ranks' experts map to `capacity`: outside [0, capacity), so the routing plan drops them
        slot_idx = table[torch.where(local, idx - lo, torch.full_like(idx, self.experts)).long()].contiguous()
        return experts_forward(x, slot_idx, wts, self.w13, self.w2, 0, swiglu_limit, base)
