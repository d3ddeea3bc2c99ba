"""Front-ends of the differential-attention kernels: per-head query / key norm prologue with a position-dependent query
temperature (csrc/kernels/qk_head_prep.cu), prompt tiles on the tensor cores (attn_diff_prefill.cu) and single rows
(attn_diff_rows.cu).  Vectors are padded to multiples of 16 with zero rows of the projections.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from ..utils import canary
from . import _lib

_f = ctypes.c_float
NUM_SMS = 148
# entries with fewer new rows than this take the row kernel (keys of one row split over the SMs) instead of a 128-row tile
TILE_MIN_ROWS = 16


@dataclass
class DiffAttention:
    """Sizes and constants of one attention mixer with two softmax maps per head."""
    heads: int
    groups: int
    dim: int                    # values per query / key vector in the checkpoint
    d: int                      # padded
    vdim: int
    v: int                      # padded
    scale: float
    lam: float                  # weight of the second map
    diff: float
    eps: float
    q_w: torch.Tensor           # fp32 [d]
    k_w: torch.Tensor | None    # None: the keys and values are another layer's
    temp_coef: float = 0.0
    temp_every: float = 0.0     # 0: no temperature

    @property
    def q_width(self) -> int:
        return self.heads * 2 * self.d

    @property
    def k_width(self) -> int:
        return self.groups * 2 * self.d

    @property
    def v_width(self) -> int:
        return self.groups * self.v


def head_prep(proj: torch.Tensor, m: DiffAttention, positions, slots, k_cache, v_cache) -> torch.Tensor:
    """``proj`` = [q | k | v | ..] (or [q | ..] of a layer that borrows its keys): per-vector norms, query temperature, cache
    append.  Returns the queries [T, heads, 2, d] in the dtype of ``proj``."""
    t = proj.shape[0]
    own = m.k_w is not None
    assert proj.stride(1) == 1
    if own:
        assert k_cache.shape[-1] == m.k_width and v_cache.shape[-1] == m.v_width and k_cache.dtype == v_cache.dtype == proj.dtype
        _lib.check_indices(slots, 0, k_cache.numel() // m.k_width, 2)
    q = torch.empty(t, m.heads, 2, m.d, dtype=proj.dtype, device=proj.device)
    rc = _lib.lib().b200_qk_head_prep(
        _lib.ptr(proj), proj.stride(0), 0, m.q_width, m.q_width + m.k_width, m.heads * 2, m.groups * 2 if own else 0,
        m.v_width if own else 0, m.d, m.dim, _lib.ptr(m.q_w), _lib.ptr(m.k_w), _f(m.eps), _f(m.temp_coef),
        ctypes.c_double(m.temp_every), _lib.ptr(positions), _lib.ptr(slots), _lib.ptr(q), _lib.ptr(k_cache if own else None),
        _lib.ptr(v_cache if own else None), t, int(proj.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "qk_head_prep")
    return q


def tiles_supported(m: DiffAttention, block_size: int) -> bool:
    return _lib.lib().b200_attn_diff_prefill_slices(m.heads, m.groups, m.d, m.v, block_size) > 0


def prefill(q: torch.Tensor, m: DiffAttention, k_cache, v_cache, gate: torch.Tensor, block_table, q_start, q_len, kv_len,
            max_q_len: int, out: torch.Tensor, seq: torch.Tensor | None = None) -> torch.Tensor:
    """Rows of several sequences' portions (tensor-core tiles).  ``gate``: logits [rows, heads] (row stride allowed); ``out``
    [rows, ldo] bf16 in place; ``seq`` names each entry's row of ``block_table``."""
    nb, bs, _ = k_cache.shape
    rows = q.shape[0]
    _lib.check_indices(block_table, 0, nb, 3)
    slices = _lib.lib().b200_attn_diff_prefill_slices(m.heads, m.groups, m.d, m.v, bs)
    diff = torch.empty(rows, m.heads, m.v, dtype=torch.float32, device=q.device) if slices > 1 else None
    rc = _lib.lib().b200_attn_diff_prefill(
        _lib.ptr(q), _lib.ptr(k_cache), _lib.ptr(v_cache), _lib.ptr(out), _lib.ptr(diff), _lib.ptr(gate), gate.stride(0),
        _lib.ptr(block_table), _lib.ptr(seq), _lib.ptr(q_start), _lib.ptr(q_len), _lib.ptr(kv_len), q_len.numel(), int(max_q_len),
        rows, block_table.shape[1], nb, bs, m.heads, m.groups, m.d, m.v, m.vdim, out.stride(0), _f(m.scale), _f(m.lam),
        _f(1.0 - m.diff), _f(m.eps), _lib.ptr(_lib.status_word(out.device)), _lib.stream())
    _lib.check(rc, "attn_diff_prefill")
    if diff is not None:
        for lo in range(0, rows, 65535):                            # the grid's second dimension
            hi = min(rows, lo + 65535)
            rc = _lib.lib().b200_attn_diff_finish(_lib.ptr(diff[lo:hi]), _lib.ptr(out[lo:hi]), _lib.ptr(gate[lo:hi]), gate.stride(0),
                                                  hi - lo, m.heads, m.v, m.vdim, out.stride(0), _f(1.0 - m.diff), _f(m.eps),
                                                  _lib.stream())
            _lib.check(rc, "attn_diff_finish")
    return out


_ws: dict[int, torch.Tensor] = {}
_outgrown: list[torch.Tensor] = []      # smaller workspaces stay alive: captured graphs hold their addresses
WS_LIMIT = 1 << 28                      # floats of partial results per launch; more rows run in several launches


def pick_splits(rows: int, blocks_per_row: int, keys: int) -> int:
    """Slices of one row's keys: enough blocks for nearly two per SM, at least 192 keys each."""
    return max(1, min(NUM_SMS, 256 // max(1, rows * blocks_per_row), (keys + 191) // 192))


def rows(q: torch.Tensor, m: DiffAttention, k_cache, v_cache, gate: torch.Tensor, block_table, positions, max_keys: int,
         out: torch.Tensor, seq: torch.Tensor | None = None, splits: int | None = None) -> torch.Tensor:
    """Single query rows: q [B, heads, 2, d], row i at position ``positions[i]`` of the sequence in table row ``seq[i]`` (or i).
    ``max_keys``: bound on the visible keys of a row (fixes the split count).  ``out`` [B, ldo] in place."""
    b = q.shape[0]
    nb, bs, _ = k_cache.shape
    assert q.dtype == out.dtype == k_cache.dtype == gate.dtype and out.stride(1) == 1 and q.is_contiguous()
    _lib.check_indices(block_table, 0, nb, 3)
    if splits is None:
        splits = pick_splits(b, m.groups, max_keys)
    per_row = splits * m.heads * 2 * (m.v + 8)
    step = max(1, min(b, 65535, WS_LIMIT // per_row))
    dev = q.device.index or 0
    ws = _ws.get(dev)
    if ws is None or ws.numel() < step * per_row:
        if ws is not None:
            _outgrown.append(ws)
        ws = _ws[dev] = canary.empty(max(step * per_row, 1 << 20), dtype=torch.float32, device=q.device,
                                     name="differential attention partials")
    for lo in range(0, b, step):
        hi = min(b, lo + step)
        rc = _lib.lib().b200_attn_diff_rows(
            _lib.ptr(q[lo:hi]), _lib.ptr(k_cache), _lib.ptr(v_cache), _lib.ptr(out[lo:hi]), _lib.ptr(gate[lo:hi]), gate.stride(0),
            _lib.ptr(block_table if seq is not None else block_table[lo:hi]), _lib.ptr(None if seq is None else seq[lo:hi]),
            _lib.ptr(positions[lo:hi]), _lib.ptr(ws), hi - lo, block_table.shape[1], bs, m.heads, m.groups, m.d, m.v, m.vdim,
            int(splits), out.stride(0), _f(m.scale), _f(m.lam), _f(1.0 - m.diff), _f(m.eps), int(out.dtype == torch.float32),
            _lib.stream())
        _lib.check(rc, "attn_diff_rows", 2)
    return out
