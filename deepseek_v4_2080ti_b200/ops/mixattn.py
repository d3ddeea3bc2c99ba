"""Front-ends of the kernels for decoders with norms around each sublayer, an fp32 residual stream and attention whose
scores are mixed across heads before the softmax (csrc/kernels/residual_norm.cu, bias_act.cu, qk_row_prep.cu,
attn_mix_prefill.cu, attn_mix_rows.cu, gemm_f32.cu).

All of them exist for bf16 and for fp32 activations; the tensors' dtype decides.  Row widths are padded to multiples of
16 (``pad16``) with zero columns, head widths to multiples of 8 with zero rows of the projections, so that every access
is a full vector.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from ..utils import canary
from . import _lib

_f = ctypes.c_float
_ll = ctypes.c_longlong
NUM_SMS = 148
# entries with fewer new rows than this take the row kernel (keys of one row split over the SMs) instead of a 128-row tile
TILE_MIN_ROWS = 16


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
    def make(w: torch.Tensor, dtype: torch.dtype, device, pad_n: bool = True) -> "Projection":
        from .gemm import PackedLinear
        n, k = w.shape
        np_, kp = pad16(n) if pad_n else n, pad16(k)
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

    def bias_xielu(self, x: torch.Tensor, bias: torch.Tensor, ap: float, an: float) -> torch.Tensor:
        """xIELU(projection + bias): in the GEMM's epilogue, or as a second kernel in fp32."""
        if self.w32 is None:
            from . import gemm
            return gemm.linear_bias_xielu(x, self.packed, bias, ap, an)
        return bias_xielu(gemm_f32(x, self.w32), bias, ap, an)

    def nbytes(self) -> int:
        return self.n * self.k * (4 if self.packed is None else 2)


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
                  unit_offset: bool = False, write_x: bool = True) -> torch.Tensor | None:
    """One boundary between sublayers of an fp32 residual ``x`` [T, ld] (updated in place):
    ``x += norm(delta + bias) * post_w``, ``x += step``, and the return value ``norm(x) * pre_w`` in ``dtype`` (None
    without ``pre_w``).  ``ids`` / ``table``: the row starts as an embedding row instead of ``x``.  ``rows`` (int32):
    only these rows are processed, and ``x`` is left alone.  Layer norm, or RMS norm with ``rms``."""
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
    out = torch.empty(n, ld, dtype=dtype, device=x.device) if pre_w is not None else None
    rc = _lib.lib().b200_residual_norm(
        _lib.ptr(x), _lib.ptr(ids), _lib.ptr(table), 0 if table is None else table.shape[0], _lib.ptr(delta), _lib.ptr(bias),
        _lib.ptr(post_w), _lib.ptr(step), _lib.ptr(pre_w), _lib.ptr(out), _lib.ptr(rows), n, ld, cols, _f(eps), int(rms),
        int(unit_offset), int(write_x and rows is None), int(dtype == torch.float32), _lib.stream())
    _lib.check(rc, "residual_norm")
    return out


def bias_xielu(z: torch.Tensor, bias: torch.Tensor | None, ap: float, an: float) -> torch.Tensor:
    """xIELU(z + bias) with the positive-side and negative-side coefficients."""
    out = torch.empty_like(z)
    rc = _lib.lib().b200_bias_xielu(_lib.ptr(z), _lib.ptr(bias), _lib.ptr(out), _ll(z.shape[0]), z.shape[1], _f(ap), _f(an),
                                    int(z.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "bias_xielu")
    return out


# ---------------------------------------------------------------------------------------------- rotary tables
def yarn_freqs(dims: int, base: float, scaling: dict | None, device) -> tuple[torch.Tensor, float]:
    """(fp64 frequencies [dims / 2], factor on cosine and sine) of an interleaved rotary embedding, with the YaRN ramp
    between the scaled and the plain frequencies when ``scaling`` (factor, original, fast, slow) is given."""
    f = base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / max(dims, 1))
    if not scaling:
        return f.to(device), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])
    turn_dim = lambda turns: dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(turn_dim(float(scaling["fast"]))), 0)
    hi = min(math.ceil(turn_dim(float(scaling["slow"]))), dims - 1)
    ramp = ((torch.arange(dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
    return (f / factor * ramp + f * (1 - ramp)).to(device), 0.1 * math.log(factor) + 1.0


# ---------------------------------------------------------------------------------------------- attention
@dataclass
class HeadMix:
    """Sizes and constants of one attention mixer."""
    heads: int
    groups: int
    dim: int                    # values per head in the checkpoint
    d: int                      # padded head width (multiple of 8)
    scale: float
    chunk: int                  # positions per chunk, 0: plain causal
    rot: int
    freq: torch.Tensor          # fp64 [rot / 2]
    mscale: float
    eps: float
    q_w: torch.Tensor           # fp32 [heads * d], [groups * d]
    k_w: torch.Tensor
    talk_t: torch.Tensor        # fp32 [heads (g), pad4(heads) (h)]


def qk_row_prep(proj: torch.Tensor, m: HeadMix, positions, slots, k_cache, v_cache, n_mix: int):
    """Whole-row QK norm, interleaved rotation and cache append of ``proj`` = [q | k]; the raw key columns are the
    values.  Returns (q_mix [n_mix, H, G * d] bf16 or None, q_row [T - n_mix, H, d] fp32 or None)."""
    t, dev = proj.shape[0], proj.device
    kw = m.groups * m.d
    assert k_cache.shape[-1] == kw and k_cache.dtype == proj.dtype and k_cache.is_contiguous() and v_cache.is_contiguous()
    _lib.check_indices(slots, 0, k_cache.numel() // kw, 2)
    q_mix = torch.empty(n_mix, m.heads, kw, dtype=torch.bfloat16, device=dev) if n_mix else None
    q_row = torch.empty(t - n_mix, m.heads, m.d, dtype=torch.float32, device=dev) if n_mix < t else None
    q_off, k_off = 0, m.heads * m.d
    rc = _lib.lib().b200_qk_row_prep(
        _lib.ptr(proj), proj.stride(0), q_off, k_off, k_off, _lib.ptr(m.q_w), _lib.ptr(m.k_w), m.heads * m.dim,
        m.groups * m.dim, _f(m.eps), _lib.ptr(m.freq), m.rot, _f(m.mscale), _lib.ptr(m.talk_t), _lib.ptr(positions),
        _lib.ptr(slots), _lib.ptr(q_mix), _lib.ptr(q_row), _lib.ptr(k_cache), _lib.ptr(v_cache), t, n_mix, m.heads, m.groups,
        m.d, int(proj.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "qk_row_prep")
    return q_mix, q_row


def tiles_supported(m: HeadMix, block_size: int) -> bool:
    return bool(_lib.lib().b200_attn_mix_prefill_supported(m.heads, m.groups, m.d, block_size))


def prefill(q_mix: torch.Tensor, m: HeadMix, k_cache, v_cache, block_table, q_start, q_len, kv_len, max_q_len: int,
            out: torch.Tensor, seq: torch.Tensor | None = None) -> torch.Tensor:
    """Rows of several sequences' portions (tensor-core tiles).  ``out`` [rows, ldo] bf16 is written in place; ``seq``
    names each entry's row of ``block_table``."""
    nb, bs, _ = k_cache.shape
    _lib.check_indices(block_table, 0, nb, 3)
    rc = _lib.lib().b200_attn_mix_prefill(
        _lib.ptr(q_mix), _lib.ptr(k_cache), _lib.ptr(v_cache), _lib.ptr(out), _lib.ptr(block_table), _lib.ptr(seq),
        _lib.ptr(q_start), _lib.ptr(q_len), _lib.ptr(kv_len), q_len.numel(), int(max_q_len), q_mix.shape[0],
        block_table.shape[1], nb, bs, m.heads, m.groups, m.d, m.chunk, out.stride(0), _f(m.scale),
        _lib.ptr(_lib.status_word(out.device)), _lib.stream())
    _lib.check(rc, "attn_mix_prefill")
    return out


_ws: dict[int, torch.Tensor] = {}
_outgrown: list[torch.Tensor] = []      # smaller workspaces stay alive: captured graphs hold their addresses


def pick_splits(rows: int, keys: int) -> int:
    """Slices of one row's keys: enough blocks for two per SM, at least 64 keys each."""
    return max(1, min(NUM_SMS, (2 * NUM_SMS) // max(1, rows), (keys + 63) // 64))


def rows(q: torch.Tensor, m: HeadMix, k_cache, v_cache, block_table, positions, max_keys: int, out: torch.Tensor,
         seq: torch.Tensor | None = None, splits: int | None = None) -> torch.Tensor:
    """Single query rows: q [B, H, d] fp32, row i at position ``positions[i]`` of the sequence in table row ``seq[i]``
    (or i).  ``max_keys``: bound on the visible keys of a row (fixes the split count).  ``out`` [B, ldo] in place."""
    b = q.shape[0]
    nb, bs, _ = k_cache.shape
    assert out.dtype == k_cache.dtype and out.stride(1) == 1
    _lib.check_indices(block_table, 0, nb, 3)
    if splits is None:
        splits = pick_splits(b, max_keys)
    ws = None
    if splits > 1:
        need = b * splits * m.heads * (m.d + 8)
        dev = q.device.index or 0
        ws = _ws.get(dev)
        if ws is None or ws.numel() < need:
            if ws is not None:
                _outgrown.append(ws)
            ws = _ws[dev] = canary.empty(max(need, 1 << 20), dtype=torch.float32, device=q.device,
                                         name="mixed-head attention partials")
    f32 = int(out.dtype == torch.float32)
    for lo in range(0, b, 65535):                                   # the grid's second dimension
        hi = min(b, lo + 65535)
        rc = _lib.lib().b200_attn_mix_rows(
            _lib.ptr(q[lo:hi]), _lib.ptr(k_cache), _lib.ptr(v_cache), _lib.ptr(out[lo:hi]), _lib.ptr(m.talk_t),
            _lib.ptr(block_table if seq is not None else block_table[lo:hi]), _lib.ptr(None if seq is None else seq[lo:hi]),
            _lib.ptr(positions[lo:hi]), _lib.ptr(ws), hi - lo, block_table.shape[1], bs, m.heads, m.groups, m.d, m.chunk,
            int(splits), out.stride(0), _f(m.scale), f32, _lib.stream())
        _lib.check(rc, "attn_mix_rows", 2 if splits > 1 else 1)
    return out
