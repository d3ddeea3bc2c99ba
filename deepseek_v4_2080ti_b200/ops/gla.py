"""Front-ends of gated linear attention (csrc/kernels/gated_linear.cu, gla_chunk.cu): decay per key channel from low-rank
logits, recurrence over a batch of rows of several sequences (``ops.scan.Segments``), per-head norm and gate.  Batches of
single rows are one launch; bf16 portions run in chunks on the tensor cores, fp32 and very short portions token by token."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib

_f = ctypes.c_float
CHUNK_MIN_ROWS = 16             # bf16 portions with fewer rows run token by token
STEP_MAX_V = 1024               # widest value head of the single-row kernel


@dataclass
class GatedLinear:
    """Sizes and constants of one mixer (``d``, ``v``, ``rank``: padded)."""
    heads: int
    dim: int
    d: int
    vdim: int
    v: int
    tau: float
    eps: float
    rank: int
    w2: torch.Tensor            # [heads * d, rank] in the activations' type
    b2: torch.Tensor            # fp32 [heads * d]
    norm_w: torch.Tensor        # fp32 [v]

    @property
    def offsets(self) -> tuple[int, int, int, int, int]:
        """Columns of q, k, v, gate and decay latent in the projection."""
        hd, hv = self.heads * self.d, self.heads * self.v
        return 0, hd, 2 * hd, 2 * hd + hv, 2 * hd + 2 * hv


def recurrence(proj: torch.Tensor, m: GatedLinear, state: torch.Tensor, seg, positions, ldo: int) -> torch.Tensor:
    """``proj`` [T, >= columns of m.offsets]; ``state`` fp32 [slots, heads, d, v], updated in place.  Returns the normalised and
    gated rows [T, ldo] (zero columns behind the heads)."""
    t = proj.shape[0]
    f32 = int(proj.dtype == torch.float32)
    assert proj.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (m.heads, m.d, m.v)
    _lib.check_indices(seg.slot, 0, state.shape[0], 4)
    L, dev = _lib.lib(), proj.device
    q, k, v, g, a = (proj[:, o:] for o in m.offsets)
    ld = proj.stride(0)
    scale, entries = m.dim ** -0.5, seg.first.numel()
    if seg.max_length == 1 and m.v <= STEP_MAX_V:
        out = torch.empty(t, ldo, dtype=proj.dtype, device=dev)
        rc = L.b200_gla_step(_lib.ptr(q), _lib.ptr(k), _lib.ptr(v), _lib.ptr(g), _lib.ptr(a), ld, _lib.ptr(m.w2), _lib.ptr(m.b2),
                             _f(1.0 / m.tau), m.rank, _lib.ptr(state), _lib.ptr(seg.first), _lib.ptr(seg.slot), _lib.ptr(positions),
                             entries, m.heads, m.d, m.v, m.vdim, _f(scale), _lib.ptr(m.norm_w), _f(m.eps), _lib.ptr(out), ldo, f32,
                             _lib.stream())
        _lib.check(rc, "gla_step")
        return out
    la = torch.empty(t, m.heads * m.d, dtype=torch.float32, device=dev)
    rc = L.b200_gla_decay(_lib.ptr(a), ld, _lib.ptr(m.w2), _lib.ptr(m.b2), _f(1.0 / m.tau), _lib.ptr(la), t, m.heads * m.d, m.rank, f32,
                          _lib.stream())
    _lib.check(rc, "gla_decay")
    o = torch.empty(t, m.heads * m.v, dtype=torch.float32, device=dev)
    rows = 0 if f32 else L.b200_gla_chunk_rows(m.d)
    chunked = rows > 0 and seg.max_length >= CHUNK_MIN_ROWS
    if chunked:
        chunks = t // rows + entries
        ws = torch.empty(chunks * m.heads * L.b200_gla_chunk_ws(m.d), dtype=torch.bfloat16, device=dev)
        end = torch.empty(chunks * m.heads * L.b200_gla_chunk_end(m.d), dtype=torch.float32, device=dev)
        rc = L.b200_gla_chunk(_lib.ptr(q), _lib.ptr(k), _lib.ptr(v), ld, _lib.ptr(la), _lib.ptr(state), _lib.ptr(o),
                              _lib.ptr(seg.first), _lib.ptr(seg.length), _lib.ptr(seg.slot), _lib.ptr(positions), entries,
                              CHUNK_MIN_ROWS, chunks, _lib.ptr(ws), _lib.ptr(end), m.heads, m.d, m.v, _f(scale), _lib.stream())
        _lib.check(rc, "gla_chunk", 2)
    if not chunked or seg.min_length < CHUNK_MIN_ROWS:
        rc = L.b200_gla_scan(_lib.ptr(q), _lib.ptr(k), _lib.ptr(v), ld, _lib.ptr(la), _lib.ptr(state), _lib.ptr(o),
                             _lib.ptr(seg.first), _lib.ptr(seg.length), _lib.ptr(seg.slot), _lib.ptr(positions), entries,
                             CHUNK_MIN_ROWS - 1 if chunked else 0, m.heads, m.d, m.v, _f(scale), f32, _lib.stream())
        _lib.check(rc, "gla_scan")
    out = torch.empty(t, ldo, dtype=proj.dtype, device=dev)
    rc = L.b200_gla_finish(_lib.ptr(o), _lib.ptr(g), ld, _lib.ptr(m.norm_w), _lib.ptr(out), ldo, t, m.heads, m.v, m.vdim, _f(m.eps), f32,
                           _lib.stream())
    _lib.check(rc, "gla_finish")
    return out
