"""Front-ends of the recurrences with one decay per head (csrc/kernels/decay_rule.cu, retention_chunk.cu,
delta_chunk.cu): retention (a fixed decay, rotated queries and keys) and the gated delta rule, each over a batch of rows of several sequences (``ops.scan.Segments``),
with per-head norm and gate.  Batches of single rows are one launch; bf16 portions run in chunks on the tensor cores, fp32 and
very short portions token by token."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from ..utils import canary
from . import _lib, scan

_f = ctypes.c_float
CHUNK_MIN_ROWS = 16             # bf16 portions with fewer rows run token by token
STEP_MAX_V = 2048               # widest value head of the single-row kernel


@dataclass
class Retention:
    """Sizes and constants of one mixer (``d``, ``v``: padded).  Its projection holds [q | k | v | gate]."""
    heads: int
    dim: int
    d: int
    vdim: int
    v: int
    eps: float
    rot: int
    freq: torch.Tensor          # fp64 [rot / 2]
    decay: torch.Tensor         # fp32 [heads]
    log2_decay: torch.Tensor    # fp32 [heads]
    norm_w: torch.Tensor        # fp32 [v]

    @property
    def width(self) -> int:
        return 2 * self.heads * (self.d + self.v)


@dataclass
class DeltaRule:
    """Sizes and constants of one mixer (``d``, ``v``: padded).  Its projection holds [q | k | v | gate | a | b]; the first
    three go through the convolution."""
    heads: int
    groups: int                 # query / key heads
    dim: int
    d: int
    vdim: int
    v: int
    eps: float
    conv: torch.Tensor          # fp32 [taps, channels]
    neg_a: torch.Tensor         # fp32 [heads] -exp(A)
    dt: torch.Tensor            # fp32 [heads]
    norm_w: torch.Tensor        # fp32 [v]

    @property
    def channels(self) -> int:
        return 2 * self.groups * self.d + self.heads * self.v


_ws: dict[int, torch.Tensor] = {}


def _workspace(sizes: list[int], device) -> list[int]:
    """Addresses of buffers of the given bytes in the device's workspace (used within one call; grown on demand)."""
    sizes = [(n + 255) // 256 * 256 for n in sizes]
    dev = device.index or 0
    ws = _ws.get(dev)
    if ws is None or ws.numel() < sum(sizes):
        ws = _ws[dev] = canary.empty(max(sum(sizes), 1 << 20), dtype=torch.uint8, device=device, name="recurrence chunks")
    out, at = [], ws.data_ptr()
    for n in sizes:
        out.append(ctypes.c_void_p(at))
        at += n
    return out


def _scan(q, k, v, log_decay, decay, beta, m, groups: int, state, o, seg, positions, max_len: int) -> None:
    rc = _lib.lib().b200_decay_scan(_lib.ptr(q), _lib.ptr(k), _lib.ptr(v), v.stride(0), _lib.ptr(log_decay), _lib.ptr(decay), _lib.ptr(beta),
                                    _lib.ptr(state), _lib.ptr(o), _lib.ptr(seg.first), _lib.ptr(seg.length), _lib.ptr(seg.slot),
                                    _lib.ptr(positions), seg.first.numel(), max_len, m.heads, groups, m.d, m.v,
                                    int(v.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "decay_scan")


def _delta_portions(q, k, v, log_decay, beta, m: "DeltaRule", state, seg, positions) -> torch.Tensor:
    """Prepared rows -> read-outs fp32 [T, heads * v]; ``state`` in place."""
    t, dev, L, entries = v.shape[0], v.device, _lib.lib(), seg.first.numel()
    o = torch.empty(t, m.heads * m.v, dtype=torch.float32, device=dev)
    n = 0 if v.dtype == torch.float32 else L.b200_delta_chunk_rows(m.d)
    chunked = n > 0 and seg.max_length >= CHUNK_MIN_ROWS
    if chunked:
        chunks, w = t // n + entries, L.b200_delta_chunk_width(m.d)
        rows, mats, fade = _workspace([chunks * m.groups * 8 * n * w, chunks * m.heads * 8 * n * n, chunks * m.heads * 8 * n], dev)
        rc = L.b200_delta_chunk(_lib.ptr(q), _lib.ptr(k), _lib.ptr(v), v.stride(0), _lib.ptr(log_decay), _lib.ptr(beta), _lib.ptr(state),
                                _lib.ptr(o), _lib.ptr(seg.first), _lib.ptr(seg.length), _lib.ptr(seg.slot), _lib.ptr(positions), entries,
                                CHUNK_MIN_ROWS, chunks, rows, mats, fade, m.heads, m.groups, m.d, m.v, _lib.stream())
        _lib.check(rc, "delta_chunk", 2)
    if not chunked or seg.min_length < CHUNK_MIN_ROWS:
        _scan(q, k, v, log_decay, None, beta, m, m.groups, state, o, seg, positions, CHUNK_MIN_ROWS - 1 if chunked else 0)
    return o


def _retention_portions(q, k, v, m: "Retention", state, seg, positions) -> torch.Tensor:
    """Prepared rows -> read-outs fp32 [T, heads * v]; ``state`` in place."""
    t, dev, L, entries = v.shape[0], v.device, _lib.lib(), seg.first.numel()
    o = torch.empty(t, m.heads * m.v, dtype=torch.float32, device=dev)
    n = 0 if v.dtype == torch.float32 else L.b200_retention_chunk_rows(m.d)
    chunked = n > 0 and seg.max_length >= CHUNK_MIN_ROWS
    if chunked:
        chunks = t // n + entries
        ws, end = _workspace([chunks * m.heads * L.b200_retention_chunk_ws(m.d) * 2, chunks * m.heads * 4], dev)
        rc = L.b200_retention_chunk(_lib.ptr(q), _lib.ptr(k), _lib.ptr(v), v.stride(0), _lib.ptr(m.log2_decay), _lib.ptr(state), _lib.ptr(o),
                                    _lib.ptr(seg.first), _lib.ptr(seg.length), _lib.ptr(seg.slot), _lib.ptr(positions), entries,
                                    CHUNK_MIN_ROWS, chunks, ws, end, m.heads, m.d, m.v, _lib.stream())
        _lib.check(rc, "retention_chunk", 2)
    if not chunked or seg.min_length < CHUNK_MIN_ROWS:
        _scan(q, k, v, None, m.decay, None, m, m.heads, state, o, seg, positions, CHUNK_MIN_ROWS - 1 if chunked else 0)
    return o


def _finish(o: torch.Tensor, gate: torch.Tensor, m, ldo: int) -> torch.Tensor:
    t = gate.shape[0]
    out = torch.empty(t, ldo, dtype=gate.dtype, device=gate.device)
    rc = _lib.lib().b200_gla_finish(_lib.ptr(o), _lib.ptr(gate), gate.stride(0), _lib.ptr(m.norm_w), _lib.ptr(out), ldo, t, m.heads, m.v,
                                    m.vdim, _f(m.eps), int(gate.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "gla_finish")
    return out


def _check(m, state, seg, proj) -> None:
    assert proj.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (m.heads, m.d, m.v)
    _lib.check_indices(seg.slot, 0, state.shape[0], 4)


def retention(proj: torch.Tensor, m: Retention, state: torch.Tensor, seg, positions, ldo: int) -> torch.Tensor:
    """``proj`` [T, >= m.width]; ``state`` fp32 [slots, heads, d, v], updated in place.  Returns the normalised and gated rows
    [T, ldo] (zero columns behind the heads)."""
    _check(m, state, seg, proj)
    t, hd, hv, ld = proj.shape[0], m.heads * m.d, m.heads * m.v, proj.stride(0)
    q, k, v, g = proj, proj[:, hd:], proj[:, 2 * hd:], proj[:, 2 * hd + hv:]
    f32, dev, scale = int(proj.dtype == torch.float32), proj.device, m.dim ** -0.5
    if seg.max_length == 1 and m.v <= STEP_MAX_V:
        out = torch.empty(t, ldo, dtype=proj.dtype, device=dev)
        rc = _lib.lib().b200_decay_step(
            _lib.ptr(q), _lib.ptr(k), _lib.ptr(v), ld, _lib.ptr(g), _lib.ptr(None), _lib.ptr(None), ld, _lib.ptr(None), _lib.ptr(None),
            _lib.ptr(m.decay), _lib.ptr(m.freq), m.rot, _lib.ptr(state), _lib.ptr(seg.first), _lib.ptr(seg.slot), _lib.ptr(positions),
            seg.first.numel(), m.heads, m.heads, m.d, m.v, m.vdim, _f(scale), _lib.ptr(m.norm_w), _f(m.eps), _lib.ptr(out), ldo, f32,
            _lib.stream())
        _lib.check(rc, "decay_step")
        return out
    qf, kf = (torch.empty(t, hd, dtype=torch.float32, device=dev) for _ in range(2))
    rc = _lib.lib().b200_rotate_prep(_lib.ptr(q), _lib.ptr(k), ld, _lib.ptr(positions), _lib.ptr(m.freq), m.rot, _f(scale), _lib.ptr(qf),
                                     _lib.ptr(kf), t, m.heads, m.d, f32, _lib.stream())
    _lib.check(rc, "rotate_prep")
    return _finish(_retention_portions(qf, kf, v, m, state, seg, positions), g, m, ldo)


def delta_rule(proj: torch.Tensor, m: DeltaRule, state: torch.Tensor, tail: torch.Tensor, seg, positions, ldo: int) -> torch.Tensor:
    """``proj`` [T, >= m.channels + heads * v + 2 heads]; ``state`` fp32 [slots, heads, d, v] and ``tail`` [slots, taps - 1,
    channels] are updated in place.  Returns the normalised and gated rows [T, ldo] (zero columns behind the heads)."""
    _check(m, state, seg, proj)
    t, gd, c = proj.shape[0], m.groups * m.d, m.channels
    g, a = proj[:, c:], proj[:, c + m.heads * m.v:]
    b = a[:, m.heads:]
    f32, dev, scale, ldg = int(proj.dtype == torch.float32), proj.device, m.dim ** -0.5, proj.stride(0)
    x = scan.conv_rows(proj, m.conv, None, tail, seg, positions)
    if seg.max_length > 1 and m.conv.shape[0] > 1:
        scan.conv_tails(proj, tail, seg)
    if seg.max_length == 1 and m.v <= STEP_MAX_V:
        out = torch.empty(t, ldo, dtype=proj.dtype, device=dev)
        rc = _lib.lib().b200_decay_step(
            _lib.ptr(x), _lib.ptr(x[:, gd:]), _lib.ptr(x[:, 2 * gd:]), c, _lib.ptr(g), _lib.ptr(a), _lib.ptr(b), ldg, _lib.ptr(m.neg_a),
            _lib.ptr(m.dt), _lib.ptr(None), _lib.ptr(None), 0, _lib.ptr(state), _lib.ptr(seg.first), _lib.ptr(seg.slot),
            _lib.ptr(positions), seg.first.numel(), m.heads, m.groups, m.d, m.v, m.vdim, _f(scale), _lib.ptr(m.norm_w), _f(m.eps),
            _lib.ptr(out), ldo, f32, _lib.stream())
        _lib.check(rc, "decay_step")
        return out
    qf, kf = (torch.empty(t, gd, dtype=torch.float32, device=dev) for _ in range(2))
    ld_, beta = (torch.empty(t, m.heads, dtype=torch.float32, device=dev) for _ in range(2))
    rc = _lib.lib().b200_delta_prep(_lib.ptr(x), c, _lib.ptr(a), _lib.ptr(b), ldg, _lib.ptr(m.neg_a), _lib.ptr(m.dt), _lib.ptr(qf),
                                    _lib.ptr(kf), _lib.ptr(ld_), _lib.ptr(beta), t, m.heads, m.groups, m.d, _f(scale), f32, _lib.stream())
    _lib.check(rc, "delta_prep")
    return _finish(_delta_portions(qf, kf, x[:, 2 * gd:], ld_, beta, m, state, seg, positions), g, m, ldo)
