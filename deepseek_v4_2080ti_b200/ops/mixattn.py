"""Front-ends of the attention kernels whose scores are mixed across heads before the softmax
(csrc/kernels/qk_row_prep.cu, attn_mix_prefill.cu, attn_mix_rows.cu).

All of them exist for bf16 and for fp32 activations; the tensors' dtype decides.  Head widths are padded to multiples of 8
with zero rows of the projections, so that every access is a full vector.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from ..utils import canary
from . import _lib
from .decoder import Projection, bias_xielu, gemm_f32, pad8, pad16, residual_norm  # noqa: F401 (part of this seam)

_f = ctypes.c_float
NUM_SMS = 148
# entries with fewer new rows than this take the row kernel (keys of one row split over the SMs) instead of a 128-row tile
TILE_MIN_ROWS = 16


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
