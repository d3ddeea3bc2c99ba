"""Pieces shared by the decoders with an fp32 residual stream: padded projections, the boundary between sublayers
(csrc/kernels/residual_norm.cu), activations (bias_act.cu) and the fp32 GEMM (gemm_f32.cu).

All of them exist for bf16 and for fp32 activations; the tensors' dtype decides.  Row widths are padded to multiples of 16
(``pad16``) with zero columns, so that every access is a full vector.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib

_f = ctypes.c_float
_ll = ctypes.c_longlong


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


# ---------------------------------------------------------------------------------------------- projections
@dataclass
class Projection:
    """[N, K] weight with both sides padded to multiples of 16 by zeros: bf16 for the tensor-core GEMM, fp32 for the
    fp32 one."""
    packed: object              # PackedLinear, or None
    w32: torch.Tensor | None
    n: int
    k: int

    @staticmethod
    def make(w: torch.Tensor, dtype: torch.dtype, device, pad_n: bool = True, tile_n: bool = False) -> "Projection":
        """``tile_n``: rows up to a multiple of 256 where that adds at most an eighth, so that prefill-sized batches tile
        evenly on the CTA-pair GEMM."""
        from .gemm import PackedLinear
        n, k = w.shape
        np_, kp = pad16(n) if pad_n else n, pad16(k)
        if pad_n and tile_n and (n + 255) // 256 * 256 <= n + n // 8:
            np_ = (n + 255) // 256 * 256
        full = torch.zeros(np_, kp, dtype=dtype, device=device)
        full[:n, :k] = w.to(device, dtype)
        if dtype == torch.float32:
            return Projection(None, full, np_, kp)
        return Projection(PackedLinear.from_bf16(full), None, np_, kp)

    def __call__(self, x: torch.Tensor, out_f32: bool = False) -> torch.Tensor:
        if self.w32 is None:
            from . import gemm
            return gemm.linear(x, self.packed, out_f32=out_f32)
        return gemm_f32(x, self.w32)

    def glu(self, x: torch.Tensor, limit: float, slope: float = 1.702) -> torch.Tensor:
        """Gated unit over this projection's [gate | up] features, which ``interleave_glu`` laid out in tiles: in the GEMM's
        epilogue where the batch tiles evenly on the CTA-pair kernel, in a kernel of its own otherwise."""
        if self.w32 is None:
            from . import gemm
            if gemm.glu_fusable(x.shape[0], self.packed):
                return gemm.linear_glu(x, self.packed, limit, slope)
        return glu(self(x), GLU_TILE, limit, slope)

    def bias_xielu(self, x: torch.Tensor, bias: torch.Tensor, ap: float, an: float) -> torch.Tensor:
        """xIELU(projection + bias): in the GEMM's epilogue, or as a second kernel in fp32."""
        if self.w32 is None:
            from . import gemm
            return gemm.linear_bias_xielu(x, self.packed, bias, ap, an)
        return bias_xielu(gemm_f32(x, self.w32), bias, ap, an)

    def part(self, lo: int, hi: int) -> "Projection":
        """The features [lo, hi) as a projection of their own (the same memory)."""
        from .gemm import PackedLinear
        if self.w32 is not None:
            return Projection(None, self.w32[lo:hi], hi - lo, self.k)
        return Projection(PackedLinear(self.packed.wfmt, self.packed.weight[lo:hi], None, hi - lo, self.k), None, hi - lo, self.k)

    def nbytes(self) -> int:
        return self.n * self.k * (4 if self.packed is None else 2)


def pad_heads(w: torch.Tensor, n: int, parts: tuple[tuple[int, int], ...]) -> torch.Tensor:
    """[n * sum(real), ...] -> [n * sum(padded), ...]: zero rows behind every (real, padded) part of every head."""
    src = w.reshape(n, sum(r for r, _ in parts), *w.shape[1:])
    out = torch.zeros(n, sum(p for _, p in parts), *w.shape[1:], dtype=w.dtype, device=w.device)
    a = b = 0
    for real, padded in parts:
        out[:, b:b + real] = src[:, a:a + real]
        a, b = a + real, b + padded
    return out.reshape(-1, *w.shape[1:])


def cat_rows(parts: list[tuple[torch.Tensor, int]]) -> torch.Tensor:
    """Matrices below one another, each padded to the given number of rows."""
    out = torch.zeros(sum(n for _, n in parts), parts[0][0].shape[1], dtype=parts[0][0].dtype, device=parts[0][0].device)
    at = 0
    for w, n in parts:
        out[at:at + w.shape[0]] = w
        at += n
    return out


GLU_TILE = 128          # features per gate / up tile of an interleaved projection


def interleave_glu(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[I, K] gate and up weights -> [2 I', K] with their rows in alternating tiles, I' = I rounded up to whole tiles (the
    zero rows give a unit of zero)."""
    n, k = gate.shape
    np_ = (n + GLU_TILE - 1) // GLU_TILE * GLU_TILE
    out = torch.zeros(np_ // GLU_TILE, 2, GLU_TILE, k, dtype=gate.dtype, device=gate.device)
    for i, w in enumerate((gate, up)):
        full = torch.zeros(np_, k, dtype=w.dtype, device=w.device)
        full[:n] = w
        out[:, i] = full.view(-1, GLU_TILE, k)
    return out.view(2 * np_, k)


def gemm_f32(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """fp32 [T, K] x [N, K]^T without any reduced-precision mode."""
    t, k = x.shape
    assert x.dtype == w.dtype == torch.float32 and x.is_contiguous() and w.is_contiguous() and w.shape[1] == k
    y = torch.empty(t, w.shape[0], dtype=torch.float32, device=x.device)
    _lib.check(_lib.lib().b200_gemm_f32(_lib.ptr(x), _lib.ptr(w), _lib.ptr(y), t, w.shape[0], k, _lib.stream()), "gemm_f32")
    return y


# ---------------------------------------------------------------------------------------------- residual stream
def residual_norm(x: torch.Tensor, cols: int, eps: float, *, delta: torch.Tensor | None = None,
                  bias: torch.Tensor | None = None, post_w: torch.Tensor | None = None, step: torch.Tensor | None = None,
                  pre_w: torch.Tensor | None = None, ids: torch.Tensor | None = None, table: torch.Tensor | None = None,
                  rows: torch.Tensor | None = None, dtype: torch.dtype | None = None, rms: bool = False,
                  unit_offset: bool = False, write_x: bool = True, table_scale: float = 1.0,
                  plain: bool = False) -> torch.Tensor | None:
    """One boundary between sublayers of an fp32 residual ``x`` [T, ld] (updated in place):
    ``x += norm(delta + bias) * post_w``, ``x += step``, and the return value ``norm(x) * pre_w`` in ``dtype`` (None
    without ``pre_w``; with ``plain``: ``x`` itself).  ``ids`` / ``table``: the row starts as an embedding row times
    ``table_scale`` instead of ``x``.  ``rows`` (int32): only these rows are processed, and ``x`` is left alone.  Layer norm,
    or RMS norm with ``rms``."""
    ld = x.shape[1]
    n = rows.numel() if rows is not None else x.shape[0]
    ref = delta if delta is not None else table
    dtype = dtype or (ref.dtype if ref is not None else torch.bfloat16)
    assert x.dtype == torch.float32 and x.is_contiguous()
    for t in (delta, table):
        assert t is None or (t.dtype == dtype and t.shape[1] == ld and t.is_contiguous())
    for t in (bias, post_w, step, pre_w):
        assert t is None or (t.dtype == torch.float32 and t.numel() == ld)
    if ids is not None:
        _lib.check_indices(ids, 0, table.shape[0], 1)
    if rows is not None:
        _lib.check_indices(rows, 0, x.shape[0], 7)
    out = torch.empty(n, ld, dtype=dtype, device=x.device) if pre_w is not None or plain else None
    rc = _lib.lib().b200_residual_norm(
        _lib.ptr(x), _lib.ptr(ids), _lib.ptr(table), 0 if table is None else table.shape[0], _lib.ptr(delta), _lib.ptr(bias),
        _lib.ptr(post_w), _lib.ptr(step), _lib.ptr(pre_w), _lib.ptr(out), _lib.ptr(rows), n, ld, cols, _f(eps), int(rms),
        int(unit_offset), int(write_x and rows is None), _f(table_scale), int(dtype == torch.float32), _lib.stream())
    _lib.check(rc, "residual_norm")
    return out


@dataclass
class Routed:
    """Routed experts' outputs of a batch, not yet summed: rows in expert order, where each (token, choice) went, its expert
    (numbers from ``experts`` on are identity experts) and its weight."""
    y: torch.Tensor             # [routes, >= ld]
    row: torch.Tensor           # int32 [T, top]
    idx: torch.Tensor           # int32 [T, top]
    weights: torch.Tensor       # fp32 [T, top]
    experts: int


def parallel_step(x: torch.Tensor | None, cols: int, weight: float, eps: float, *, ld: int, n: int, dtype: torch.dtype,
                  x_out: torch.Tensor | None = None, ids: torch.Tensor | None = None, table: torch.Tensor | None = None,
                  mix: torch.Tensor | None = None, gates: torch.Tensor | None = None, gate_b: torch.Tensor | None = None,
                  h: torch.Tensor | None = None, routed: Routed | None = None, shared: torch.Tensor | None = None,
                  shared_gate: torch.Tensor | None = None, shift: torch.Tensor | None = None, tail: torch.Tensor | None = None,
                  seg=None, positions: torch.Tensor | None = None, rows: torch.Tensor | None = None,
                  norm: bool = True) -> tuple[torch.Tensor | None, torch.Tensor | None]:
    """Step between layers whose sublayers run side by side (csrc/kernels/parallel_step.cu):
    ``x + mix sigmoid(gates[:, :ld] + b) + ff sigmoid(gates[:, ld:] + b)`` goes to ``x_out`` (which may be ``x``), with ``ff``
    the sum of the routed experts, of identity experts (``h``) and of ``shared`` behind its gate (a column of logits).  Returns (RMS norm of it times ``weight``, that norm moved towards the row before it by ``shift``): the second
    only with ``shift``, which also keeps the sequences' ``tail`` [slots, ld].  ``rows``: only these rows, norm only."""
    dev = (x if x is not None else ids).device
    assert x is None or (x.dtype == torch.float32 and x.shape[1] == ld and x.is_contiguous())
    for t in (mix, h, shared, table):
        assert t is None or (t.dtype == dtype and t.shape[1] == ld and t.is_contiguous())
    assert gates is None or (gates.dtype == dtype and gates.stride(1) == 1 and gates.shape[1] >= ld)
    if ids is not None:
        _lib.check_indices(ids, 0, table.shape[0], 1)
    if rows is not None:
        _lib.check_indices(rows, 0, x.shape[0], 7)
    if seg is not None and tail is not None:
        _lib.check_indices(seg.row_slot, 0, tail.shape[0], 4)
    count = rows.numel() if rows is not None else n
    out = torch.empty(count, ld, dtype=dtype, device=dev) if norm else None
    m = torch.empty(n, ld, dtype=dtype, device=dev) if shift is not None else None
    single = m is not None and seg.max_length == 1      # no row needs its neighbour: shift and tails in the same launch
    f32, r = int(dtype == torch.float32), routed
    rc = _lib.lib().b200_parallel_step(
        _lib.ptr(x), _lib.ptr(x_out), _lib.ptr(ids), _lib.ptr(table), 0 if table is None else table.shape[0], _lib.ptr(mix),
        _lib.ptr(gates), 0 if gates is None else gates.stride(0), _lib.ptr(gate_b), _lib.ptr(h), _lib.ptr(r.y if r else None),
        r.y.stride(0) if r else 0, _lib.ptr(r.row if r else None), _lib.ptr(r.idx if r else None),
        _lib.ptr(r.weights if r else None), r.idx.shape[1] if r else 0, r.experts if r else 0, _lib.ptr(shared),
        _lib.ptr(shared_gate), 0 if shared_gate is None else shared_gate.stride(0), _f(weight), _f(eps), _lib.ptr(out),
        _lib.ptr(m if single else None), _lib.ptr(shift), _lib.ptr(tail), _lib.ptr(seg.row_slot if single else None),
        _lib.ptr(positions), _lib.ptr(rows), count, ld, cols, f32, _lib.stream())
    _lib.check(rc, "parallel_step")
    if m is not None and not single:
        rc = _lib.lib().b200_shift_rows(_lib.ptr(out), _lib.ptr(m), _lib.ptr(shift), _lib.ptr(tail), _lib.ptr(seg.row_first),
                                        _lib.ptr(seg.row_slot), _lib.ptr(positions), _lib.ptr(seg.first), _lib.ptr(seg.length),
                                        _lib.ptr(seg.slot), seg.first.numel(), n, ld, f32, _lib.stream())
        _lib.check(rc, "shift_rows", 2)
    return out, m


def branch_step(x: torch.Tensor | None, cols: int, eps: float, *, ld: int, n: int, dtype: torch.dtype, x_out: torch.Tensor | None = None,
                ids: torch.Tensor | None = None, table: torch.Tensor | None = None,
                normed: tuple[tuple[torch.Tensor | None, torch.Tensor], ...] = (), plain: tuple[torch.Tensor, ...] = (),
                routed: Routed | None = None, copy: bool = False, weight: torch.Tensor | None = None, conv: torch.Tensor | None = None,
                tail: torch.Tensor | None = None, seg=None, positions: torch.Tensor | None = None,
                rows: torch.Tensor | None = None) -> tuple[torch.Tensor | None, torch.Tensor | None, torch.Tensor | None]:
    """Step of a residual that takes several sublayer results at once (csrc/kernels/branch_step.cu): ``x`` (zero without it) plus up
    to two ``normed`` branches (result, weight), up to two ``plain`` ones and the ``routed`` experts' sum goes to ``x_out`` (which may
    be ``x``).  ``ids`` / ``table``: the first normed branch is an embedding row (its result is None).  Returns (that sum in ``dtype``
    with ``copy``, its RMS norm times ``weight``, that norm plus its causal convolution with ``conv`` [taps, ld]): the last keeps the
    sequences' ``tail`` [slots, taps - 1, ld]; ``conv``'s last row has the 1 of the norm itself in it.  ``rows``: only these rows."""
    from . import scan
    dev = (x if x is not None else ids).device
    assert x is None or (x.dtype == torch.float32 and x.shape[1] == ld and x.is_contiguous())
    assert len(normed) <= 2 and len(plain) <= 2
    for t in [r for r, _ in normed] + list(plain) + [table]:
        assert t is None or (t.dtype == dtype and t.shape[1] == ld and t.is_contiguous())
    for w in [w for _, w in normed] + [weight]:
        assert w is None or (w.dtype == torch.float32 and w.numel() == ld)
    if ids is not None:
        _lib.check_indices(ids, 0, table.shape[0], 1)
    if rows is not None:
        _lib.check_indices(rows, 0, x.shape[0], 7)
    if conv is not None:
        _lib.check_indices(seg.row_slot, 0, tail.shape[0], 4)
    count = rows.numel() if rows is not None else n
    new = lambda m: torch.empty(m, ld, dtype=dtype, device=dev)
    c, h = new(n) if copy else None, new(count) if weight is not None else None
    single = conv is not None and seg.max_length == 1      # no row needs its neighbour: convolution and tails in the same launch
    m = new(n) if single else None
    taps = 0 if conv is None else conv.shape[0]
    b = list(normed) + [(None, None)] * (2 - len(normed))
    p = list(plain) + [None] * (2 - len(plain))
    r, f32 = routed, int(dtype == torch.float32)
    rc = _lib.lib().b200_branch_step(
        _lib.ptr(x), _lib.ptr(x_out), _lib.ptr(ids), _lib.ptr(table), 0 if table is None else table.shape[0], _lib.ptr(b[0][0]),
        _lib.ptr(b[0][1]), _lib.ptr(b[1][0]), _lib.ptr(b[1][1]), _lib.ptr(p[0]), _lib.ptr(p[1]), _lib.ptr(r.y if r else None),
        r.y.stride(0) if r else 0, _lib.ptr(r.row if r else None), _lib.ptr(r.weights if r else None), r.idx.shape[1] if r else 0,
        _lib.ptr(c), _lib.ptr(weight), _f(eps), _lib.ptr(h), _lib.ptr(m), _lib.ptr(conv if single else None),
        _lib.ptr(tail if single else None), _lib.ptr(seg.row_slot if single else None), _lib.ptr(positions if single else None), taps,
        _lib.ptr(rows), count, ld, cols, f32, _lib.stream())
    _lib.check(rc, "branch_step")
    if conv is not None and not single:
        m = scan.conv_rows(h, conv, None, tail, seg, positions, silu=False)
        if taps > 1:
            scan.conv_tails(h, tail, seg)
    return c, h, m


def poly_norm(z: torch.Tensor, cols: int, coef: tuple[float, float, float, float], eps: float, ldo: int) -> torch.Tensor:
    """``a N(z) + b N(z^2) + c N(z^3) + e`` with N over the root mean square of a row's first ``cols`` columns: [T, ldo]."""
    out = torch.empty(z.shape[0], ldo, dtype=z.dtype, device=z.device)
    a, b, c, e = coef
    rc = _lib.lib().b200_poly_norm(_lib.ptr(z), z.stride(0), _lib.ptr(out), ldo, z.shape[0], cols, _f(a), _f(b), _f(c), _f(e),
                                   _f(eps), int(z.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "poly_norm")
    return out


TOKEN_GATE_MAX_ROWS = 64        # bf16 batches up to this take the row kernel: a GEMM tile would leave all but a few SMs idle


def token_gate(x: torch.Tensor, w: Projection, table: torch.Tensor, col: int, ids: torch.Tensor) -> torch.Tensor:
    """``gelu_tanh(x W^T) * table[ids, col:col + features of W]``; short bf16 batches in one launch."""
    assert table.dtype == x.dtype and table.is_contiguous() and x.is_contiguous()
    _lib.check_indices(ids, 0, table.shape[0], 1)
    t, L = x.shape[0], _lib.lib()
    out = torch.empty(t, w.n, dtype=x.dtype, device=x.device)
    if w.w32 is None and t <= TOKEN_GATE_MAX_ROWS:
        rc = L.b200_rows_token_gate(_lib.ptr(x), x.shape[1], _lib.ptr(w.packed.weight), _lib.ptr(table), table.shape[1], col, table.shape[0],
                                    _lib.ptr(ids), _lib.ptr(out), w.n, t, w.n, w.k, _lib.stream())
        _lib.check(rc, "rows_token_gate")
        return out
    z = w(x)
    rc = L.b200_token_gate(_lib.ptr(z), z.stride(0), _lib.ptr(table), table.shape[1], col, table.shape[0], _lib.ptr(ids), _lib.ptr(out), w.n,
                           t, int(x.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "token_gate")
    return out


def bias_xielu(z: torch.Tensor, bias: torch.Tensor | None, ap: float, an: float) -> torch.Tensor:
    """xIELU(z + bias) with the positive-side and negative-side coefficients."""
    out = torch.empty_like(z)
    rc = _lib.lib().b200_bias_xielu(_lib.ptr(z), _lib.ptr(bias), _lib.ptr(out), _ll(z.shape[0]), z.shape[1], _f(ap), _f(an),
                                    int(z.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "bias_xielu")
    return out


def glu(z: torch.Tensor, tile: int, limit: float, slope: float = 1.702) -> torch.Tensor:
    """Gated unit over rows (a stride is allowed) of gate and up features interleaved in tiles of ``tile`` columns: the clamped one-plus form
    ``min(g, limit) sigmoid(slope min(g, limit)) (clamp(u, -limit, limit) + 1)``, or ``silu(g) u`` with ``limit`` 0."""
    out = torch.empty(z.shape[0], z.shape[1] // 2, dtype=z.dtype, device=z.device)
    rc = _lib.lib().b200_glu(_lib.ptr(z), z.stride(0), _lib.ptr(out), _ll(z.shape[0]), out.shape[1], tile, _f(limit), _f(slope),
                             int(z.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "glu")
    return out
