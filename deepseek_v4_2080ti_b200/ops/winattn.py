"""Front-ends of attention with a sliding window and a learned bias per head and distance: per-head query / key norm prologue
(csrc/kernels/qk_head_prep.cu), prompt tiles on the tensor cores (attn_window_prefill.cu) and single rows (attn_window_rows.cu).  Vectors are padded to multiples of 16 with zero rows of
the projections.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from ..utils import canary
from . import _lib

_f = ctypes.c_float
NUM_SMS = 148
# entries with fewer new rows than this take the row kernel (keys of one row split over the SMs) instead of a 128-row tile
TILE_MIN_ROWS = 16


@dataclass
class WindowAttention:
    """Sizes and constants of one attention mixer."""
    heads: int
    groups: int
    dim: int                    # values per query / key vector in the checkpoint
    d: int                      # padded
    vdim: int
    v: int                      # padded
    scale: float
    size: int                   # a position sees itself and the size - 1 positions before it
    eps: float
    q_w: torch.Tensor           # fp32 [d]
    k_w: torch.Tensor
    bias: torch.Tensor          # fp32 [heads, size]: what is added to a score per distance, times log2 e

    @property
    def q_width(self) -> int:
        return self.heads * self.d

    @property
    def k_width(self) -> int:
        return self.groups * self.d

    @property
    def v_width(self) -> int:
        return self.groups * self.v


def distance_buckets(size: int, rows: int, reach: int) -> torch.Tensor:
    """Row of the bias table for every distance below ``size``: one row each in the lower half, logarithmic steps from there to
    ``reach``, the last row beyond."""
    half = rows // 2
    span = math.log(reach / half)
    log = [min(rows - 1, half + math.floor(math.log(n / half) / span * (rows - half))) for n in range(half, max(size, half))]
    return torch.tensor((list(range(half)) + log)[:size], dtype=torch.long)


def distance_bias(rel: torch.Tensor, size: int, reach: int) -> torch.Tensor:
    """rel [rows, heads] -> fp32 [heads, size], times log2 e."""
    table = rel.float()[distance_buckets(size, rel.shape[0], reach).to(rel.device)]
    return (table.t().double() / math.log(2.0)).float().contiguous()


def head_prep(proj: torch.Tensor, m: WindowAttention, positions, slots, k_cache, v_cache) -> torch.Tensor:
    """``proj`` = [q | k | v | ..]: per-head norms, cache append.  Returns the queries [T, heads, d] in the dtype of ``proj``."""
    t = proj.shape[0]
    assert proj.stride(1) == 1 and k_cache.shape[-1] == m.k_width and v_cache.shape[-1] == m.v_width
    assert k_cache.dtype == v_cache.dtype == proj.dtype
    _lib.check_indices(slots, 0, k_cache.numel() // m.k_width, 2)
    q = torch.empty(t, m.heads, m.d, dtype=proj.dtype, device=proj.device)
    rc = _lib.lib().b200_qk_head_prep(
        _lib.ptr(proj), proj.stride(0), 0, m.q_width, m.q_width + m.k_width, m.heads, m.groups, m.v_width, m.d, m.dim, _lib.ptr(m.q_w),
        _lib.ptr(m.k_w), _f(m.eps), _f(0.0), ctypes.c_double(0.0), _lib.ptr(positions), _lib.ptr(slots), _lib.ptr(q), _lib.ptr(k_cache),
        _lib.ptr(v_cache), t, int(proj.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "qk_head_prep")
    return q


def tiles_supported(m: WindowAttention, block_size: int) -> bool:
    return bool(_lib.lib().b200_attn_window_prefill_supported(m.heads, m.groups, m.d, m.v, block_size))


def prefill(q: torch.Tensor, m: WindowAttention, k_cache, v_cache, block_table, q_start, q_len, kv_len, max_q_len: int,
            out: torch.Tensor, seq: torch.Tensor | None = None) -> torch.Tensor:
    """Rows of several sequences' portions (tensor-core tiles).  ``out`` [rows, ldo] bf16 in place; ``seq`` names each entry's row
    of ``block_table``."""
    nb, bs, _ = k_cache.shape
    assert q.is_contiguous() and out.stride(1) == 1
    _lib.check_indices(block_table, 0, nb, 3)
    rc = _lib.lib().b200_attn_window_prefill(
        _lib.ptr(q), _lib.ptr(k_cache), _lib.ptr(v_cache), _lib.ptr(m.bias), _lib.ptr(out), out.stride(0), _lib.ptr(block_table),
        _lib.ptr(seq), _lib.ptr(q_start), _lib.ptr(q_len), _lib.ptr(kv_len), q_len.numel(), int(max_q_len), q.shape[0],
        block_table.shape[1], nb, bs, m.heads, m.groups, m.d, m.v, m.size, _f(m.scale), _lib.ptr(_lib.status_word(out.device)),
        _lib.stream())
    _lib.check(rc, "attn_window_prefill")
    return out


_ws: dict[int, torch.Tensor] = {}
_outgrown: list[torch.Tensor] = []      # smaller workspaces stay alive: captured graphs hold their addresses
WS_LIMIT = 1 << 28                      # floats of partial results per launch; more rows run in several launches


def pick_splits(rows: int, blocks_per_row: int, keys: int) -> int:
    """Slices of one row's keys: enough blocks for nearly two per SM, at least 128 keys each."""
    return max(1, min(NUM_SMS, 256 // max(1, rows * blocks_per_row), (keys + 127) // 128))


def rows(q: torch.Tensor, m: WindowAttention, k_cache, v_cache, block_table, positions, max_keys: int, out: torch.Tensor,
         seq: torch.Tensor | None = None, splits: int | None = None) -> torch.Tensor:
    """Single query rows: q [B, heads, d], row i at position ``positions[i]`` of the sequence in table row ``seq[i]`` (or i).
    ``max_keys``: bound on the context of a row (with the window it fixes the split count).  ``out`` [B, ldo] in place."""
    b = q.shape[0]
    nb, bs, _ = k_cache.shape
    assert q.dtype == out.dtype == k_cache.dtype and out.stride(1) == 1 and q.is_contiguous()
    _lib.check_indices(block_table, 0, nb, 3)
    if splits is None:
        splits = pick_splits(b, m.groups, min(max_keys, m.size))
    per_row = splits * m.heads * (m.v + 8) if splits > 1 else 1
    step = max(1, min(b, 65535, WS_LIMIT // per_row))
    ws = None
    if splits > 1:
        dev = q.device.index or 0
        ws = _ws.get(dev)
        if ws is None or ws.numel() < step * per_row:
            if ws is not None:
                _outgrown.append(ws)
            ws = _ws[dev] = canary.empty(max(step * per_row, 1 << 20), dtype=torch.float32, device=q.device,
                                         name="window attention partials")
    for lo in range(0, b, step):
        hi = min(b, lo + step)
        rc = _lib.lib().b200_attn_window_rows(
            _lib.ptr(q[lo:hi]), _lib.ptr(k_cache), _lib.ptr(v_cache), _lib.ptr(m.bias), _lib.ptr(out[lo:hi]),
            _lib.ptr(block_table if seq is not None else block_table[lo:hi]), _lib.ptr(None if seq is None else seq[lo:hi]),
            _lib.ptr(positions[lo:hi]), _lib.ptr(ws), hi - lo, block_table.shape[1], bs, m.heads, m.groups, m.d, m.v, m.size, int(splits),
            out.stride(0), _f(m.scale), int(out.dtype == torch.float32), _lib.stream())
        _lib.check(rc, "attn_window_rows", 2 if splits > 1 else 1)
    return out
