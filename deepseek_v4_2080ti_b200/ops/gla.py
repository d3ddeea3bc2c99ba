"""Front-ends of gated linear attention (csrc/kernels/gated_linear.cu): decay per key channel from low-rank logits, recurrence
over a batch of rows of several sequences (``ops.scan.Segments``), per-head norm and gate."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib

_f = ctypes.c_float


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
    la = torch.empty(t, m.heads * m.d, dtype=torch.float32, device=dev)
    rc = L.b200_gla_decay(_lib.ptr(a), ld, _lib.ptr(m.w2), _lib.ptr(m.b2), _f(1.0 / m.tau), _lib.ptr(la), t, m.heads * m.d, m.rank, f32,
                          _lib.stream())
    _lib.check(rc, "gla_decay")
    o = torch.empty(t, m.heads * m.v, dtype=torch.float32, device=dev)
    rc = L.b200_gla_scan(_lib.ptr(q), _lib.ptr(k), _lib.ptr(v), ld, _lib.ptr(la), _lib.ptr(state), _lib.ptr(o), _lib.ptr(seg.first),
                         _lib.ptr(seg.length), _lib.ptr(seg.slot), _lib.ptr(positions), seg.first.numel(), m.heads, m.d, m.v,
                         _f(m.dim ** -0.5), f32, _lib.stream())
    _lib.check(rc, "gla_scan")
    out = torch.empty(t, ldo, dtype=proj.dtype, device=dev)
    rc = L.b200_gla_finish(_lib.ptr(o), _lib.ptr(g), ld, _lib.ptr(m.norm_w), _lib.ptr(out), ldo, t, m.heads, m.v, m.vdim, _f(m.eps), f32,
                           _lib.stream())
    _lib.check(rc, "gla_finish")
    return out
