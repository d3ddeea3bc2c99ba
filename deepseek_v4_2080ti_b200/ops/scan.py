"""Front-ends of the recurrent-mixer kernels: causal convolution over a batch of rows of several sequences
(csrc/kernels/conv_rows.cu) and the selective scan (selective_scan.cu).

A batch is described once per pass by ``Segments``: neighbouring rows of one sequence form an entry with a state slot.
State starts at zero where a row's position is 0, so a slot that is used again needs no clearing.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from ..utils import canary
from . import _lib

SLICE_ROWS = 32                 # a time slice is a multiple of this


@dataclass
class Segments:
    """int32 device tensors: per row the first row of its entry and its state slot; per entry first row, length, slot."""
    row_first: torch.Tensor
    row_slot: torch.Tensor
    first: torch.Tensor
    length: torch.Tensor
    slot: torch.Tensor
    max_length: int
    min_length: int = 1


def conv_rows(x: torch.Tensor, w_t: torch.Tensor, bias: torch.Tensor | None, tail: torch.Tensor, seg: Segments,
              positions: torch.Tensor, silu: bool = True) -> torch.Tensor:
    """x [T, >= C] (row stride allowed), w_t fp32 [taps, C], tail [slots, taps - 1, C] -> [T, C].  The tails of sequences with a
    single row are replaced here, those of longer portions by ``selective_scan`` or ``conv_tails``."""
    taps, c = w_t.shape
    t = x.shape[0]
    assert x.stride(1) == 1 and tail.dtype == x.dtype and tail.shape[1:] == (max(taps - 1, 1), c)
    _lib.check_indices(seg.row_slot, 0, tail.shape[0], 4)
    y = torch.empty(t, c, dtype=x.dtype, device=x.device)
    rc = _lib.lib().b200_conv_rows(_lib.ptr(x), x.stride(0), _lib.ptr(w_t), _lib.ptr(bias), _lib.ptr(tail), _lib.ptr(seg.row_first),
                                   _lib.ptr(seg.row_slot), _lib.ptr(positions), _lib.ptr(y), c, t, c, taps, int(silu),
                                   int(x.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "conv_rows")
    return y


def conv_tails(x: torch.Tensor, tail: torch.Tensor, seg: Segments) -> None:
    """The tails [slots, taps - 1, C] of sequences that bring more than one row, from the convolution's inputs x [T, >= C]."""
    keep, c = tail.shape[1:]
    assert x.stride(1) == 1 and tail.dtype == x.dtype and tail.is_contiguous()
    rc = _lib.lib().b200_conv_tails(_lib.ptr(x), x.stride(0), _lib.ptr(tail), _lib.ptr(seg.first), _lib.ptr(seg.length), _lib.ptr(seg.slot),
                                    seg.first.numel(), c, keep + 1, int(x.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "conv_tails")


_ws: dict[int, torch.Tensor] = {}
_outgrown: list[torch.Tensor] = []      # smaller workspaces stay alive: captured graphs hold their addresses


def _workspace(need: int, device) -> torch.Tensor:
    dev = device.index or 0
    ws = _ws.get(dev)
    if ws is None or ws.numel() < need:
        if ws is not None:
            _outgrown.append(ws)
        ws = _ws[dev] = canary.empty(max(need, 1 << 20), dtype=torch.float32, device=device, name="selective scan slices")
    return ws


def selective_scan(x: torch.Tensor, dt: torch.Tensor, bc: torch.Tensor, b_off: int, c_off: int, z: torch.Tensor, a: torch.Tensor,
                   dt_bias: torch.Tensor, d_skip: torch.Tensor, state: torch.Tensor, seg: Segments, positions: torch.Tensor,
                   x_in: torch.Tensor | None = None, tail: torch.Tensor | None = None, slices: int | None = None) -> torch.Tensor:
    """x [T, C] (after the convolution), dt fp32 [T, C] (before bias and softplus), bc rows with B and C at the given columns,
    z [T, >= C]; ``a`` fp32 [C, N] as ``scan_decay`` prepares it; state fp32 [slots, C, N], updated in place.  Returns
    ``y silu(z)`` [T, C].  ``x_in`` / ``tail``: inputs of the convolution in front, whose last rows replace the tails of the
    sequences that bring more than one row."""
    t, c = x.shape
    n = a.shape[1]
    assert dt.dtype == state.dtype == torch.float32 and state.shape[1:] == (c, n) and state.is_contiguous() and a.is_contiguous()
    assert x.is_contiguous() and dt.stride(1) == bc.stride(1) == z.stride(1) == 1 and bc.dtype == z.dtype == x.dtype
    _lib.check_indices(seg.slot, 0, state.shape[0], 4)
    entries = seg.first.numel()
    if slices is None:
        slices = _lib.lib().b200_selective_scan_slices(c, n, entries, seg.max_length)
    per = max(SLICE_ROWS, (seg.max_length + slices - 1) // slices)
    per = (per + SLICE_ROWS - 1) // SLICE_ROWS * SLICE_ROWS
    slices = (seg.max_length + per - 1) // per
    ws_state = ws_sum = None
    if slices > 1:
        ws = _workspace(entries * slices * c * (n + 1), x.device)
        ws_state, ws_sum = ws, ws[entries * slices * c * n:]
    taps = 1 if x_in is None else tail.shape[1] + 1
    out = torch.empty(t, c, dtype=x.dtype, device=x.device)
    rc = _lib.lib().b200_selective_scan(
        _lib.ptr(x), c, _lib.ptr(dt), dt.stride(0), _lib.ptr(bc), bc.stride(0), b_off, c_off, _lib.ptr(z), z.stride(0),
        _lib.ptr(out), c, _lib.ptr(a), _lib.ptr(dt_bias), _lib.ptr(d_skip), _lib.ptr(state), _lib.ptr(seg.first),
        _lib.ptr(seg.length), _lib.ptr(seg.slot), _lib.ptr(positions), _lib.ptr(x_in), 0 if x_in is None else x_in.stride(0),
        _lib.ptr(tail), taps, c, n, entries, seg.max_length, int(seg.min_length == 1), slices, per, _lib.ptr(ws_state), _lib.ptr(ws_sum), int(x.dtype == torch.float32),
        _lib.stream())
    _lib.check(rc, "selective_scan", int(seg.min_length == 1) + (0 if seg.max_length == 1 else 2 if slices > 1 else 1))
    return out


def scan_decay(a_log: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """-exp(A_log) in fp32, times log2(e) for the bf16 kernels (their exponential is a power of two)."""
    a = -torch.exp(a_log.double())
    return ((a / torch.log(torch.tensor(2.0, dtype=torch.float64, device=a.device))) if dtype == torch.bfloat16 else a).float().contiguous()
