"""Front-ends of latent attention over a paged cache of one row per token, [latent | rotated key part], shared by all heads:
prologue (csrc/kernels/latent_prep.cu), single rows in the absorbed form (attn_latent_decode.cu on the tensor cores,
attn_latent_rows.cu for other sizes and fp32; head_linear.cu), prompt tiles on
the tensor cores over keys and values expanded from the latents (attn_heads_prefill.cu).

All of it exists for bf16 and for fp32 activations; the tensors' dtype decides.  Widths are padded to multiples of 16 with
zero columns.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from ..utils import canary
from . import _lib

_f = ctypes.c_float
NUM_SMS = 148
# Entries with fewer new rows than this take the row kernel: expanding a context of C-wide latents costs each of its rows
# 2 C (d + v) products per head, once per entry, and saves 2 (2 C + r) - 2 (d + r + v) per head and query row, on faster units.
TILE_MIN_ROWS = 32
EXPANDED_LIMIT = 1 << 29                # values of expanded keys and values held at a time; more heads go in several rounds


@dataclass
class LatentAttention:
    """Sizes and constants of one mixer (``*_pad``, ``d``, ``r``, ``v``, ``c``: padded)."""
    heads: int
    dim: int
    d: int
    rot_dim: int
    r: int
    vdim: int
    v: int
    q_rank: int
    q_pad: int
    kv_rank: int
    c: int
    scale: float
    eps: float
    rot: int                    # rotated values of the key part
    freq: torch.Tensor          # fp64 [rot / 2]
    mscale: float
    q_w: torch.Tensor           # fp32 [q_pad]
    c_w: torch.Tensor | None    # fp32 [c]; None: the cache is another layer's

    @property
    def cache_width(self) -> int:
        return self.c + self.r

    @property
    def head_width(self) -> int:
        return self.d + self.r


def prep(proj: torch.Tensor, m: LatentAttention, positions, slots, cache: torch.Tensor) -> torch.Tensor:
    """``proj`` = [query latent | latent | key part] (or [query latent] of a layer that reads another layer's cache):
    norms, rotation and cache append.  Returns the normalised query latent [T, q_pad]."""
    t, own = proj.shape[0], m.c_w is not None
    assert proj.stride(1) == 1 and cache.shape[-1] == m.cache_width and cache.dtype == proj.dtype and cache.is_contiguous()
    if own:
        _lib.check_indices(slots, 0, cache.numel() // m.cache_width, 2)
    out = torch.empty(t, m.q_pad, dtype=proj.dtype, device=proj.device)
    rc = _lib.lib().b200_latent_prep(
        _lib.ptr(proj), proj.stride(0), _lib.ptr(out), m.q_rank, m.q_pad, _lib.ptr(m.q_w), _lib.ptr(cache if own else None), m.kv_rank,
        m.c, _lib.ptr(m.c_w), m.rot_dim, m.r, m.rot, _lib.ptr(m.freq), _f(m.mscale), _f(m.eps), _lib.ptr(positions), _lib.ptr(slots), t,
        int(proj.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "latent_prep")
    return out


def rotate_heads(q: torch.Tensor, m: LatentAttention, positions, out: torch.Tensor | None = None, off: int = 0) -> torch.Tensor:
    """Rotated parts of q [T, >= heads (d + r)]: in place, or to columns ``off`` of every head of ``out`` [T, heads, w]."""
    t = q.shape[0]
    dst = q if out is None else out
    head, at = (m.head_width, m.d) if out is None else (out.shape[2], off)
    assert q.stride(1) == 1 and q.shape[1] >= m.heads * m.head_width and dst.dtype == q.dtype
    rc = _lib.lib().b200_rotate_heads(_lib.ptr(q), _lib.ptr(dst), _lib.ptr(m.freq), _lib.ptr(positions), t, m.heads, q.stride(0),
                                      m.head_width, m.d, dst.stride(0), head, at, m.r, m.rot, _f(m.mscale),
                                      int(q.dtype == torch.float32), _lib.stream())
    _lib.check(rc, "rotate_heads")
    return dst


def head_linear(x: torch.Tensor, ldx: int, x_head: int, w: torch.Tensor, y: torch.Tensor, ldy: int, y_head: int, t: int) -> None:
    """y[t, h, :N] = x[t, h, :K] w[h]^T; rows ``ldx`` / ``ldy`` apart, heads ``x_head`` / ``y_head`` apart; w [H, N, K]."""
    h, n, k = w.shape
    assert x.dtype == y.dtype == w.dtype and w.is_contiguous()
    L = _lib.lib()
    if x.dtype == torch.float32:
        rc = L.b200_head_linear_f32(_lib.ptr(x), ldx, x_head, _lib.ptr(w), _lib.ptr(y), ldy, y_head, t, h, n, k, _lib.stream())
    else:
        rc = L.b200_head_linear(_lib.ptr(x), ldx, x_head, _lib.ptr(w), _lib.ptr(y), ldy, y_head, t, h, n, k, _lib.stream())
    _lib.check(rc, "head_linear")


_ws: dict[int, torch.Tensor] = {}
_outgrown: list[torch.Tensor] = []      # smaller workspaces stay alive: captured graphs hold their addresses
WS_LIMIT = 1 << 28                      # floats of partial results per launch; more rows run in several launches


def pick_splits(blocks: int, keys: int) -> int:
    """Slices of one row's keys: enough blocks for about two per SM, at least 128 keys each."""
    return max(1, min(NUM_SMS, 2 * NUM_SMS // max(1, blocks), (keys + 127) // 128))


def attend_rows(q: torch.Tensor, m: LatentAttention, cache: torch.Tensor, block_table, positions, max_keys: int,
                seq: torch.Tensor | None = None, splits: int | None = None, tiles: bool = True) -> torch.Tensor:
    """Absorbed queries q [B, heads, c + r] of single rows, row i at position ``positions[i]`` of the sequence in table row
    ``seq[i]`` (or i) -> summed latents [B, heads, c].  ``max_keys``: bound on the visible keys of a row.  ``tiles`` False:
    not on the tcgen05 kernel, whatever the sizes."""
    b = q.shape[0]
    nb, bs, _ = cache.shape
    f32 = int(q.dtype == torch.float32)
    assert q.is_contiguous() and q.shape[1:] == (m.heads, m.cache_width) and q.dtype == cache.dtype
    _lib.check_indices(block_table, 0, nb, 3)
    out = torch.empty(b, m.heads, m.c, dtype=q.dtype, device=q.device)
    L = _lib.lib()
    group = 0 if f32 or not tiles else L.b200_attn_latent_decode_heads(m.heads, m.c, m.cache_width, bs)
    if splits is None:
        per = group or L.b200_attn_latent_rows_heads(m.heads, m.c, m.cache_width, b, f32)
        blocks = b * ((m.heads + per - 1) // per)
        # one tcgen05 CTA fills an SM; the other kernels want two blocks or more
        splits = max(1, min(NUM_SMS // blocks, (max_keys + 127) // 128)) if group else pick_splits(blocks, max_keys)
    per_row = splits * m.heads * (m.c + 2) if splits > 1 else 0
    step = min(b, 65535, WS_LIMIT // per_row if per_row else b)
    ws = None
    if splits > 1:
        dev = q.device.index or 0
        ws = _ws.get(dev)
        if ws is None or ws.numel() < step * per_row:
            if ws is not None:
                _outgrown.append(ws)
            ws = _ws[dev] = canary.empty(max(step * per_row, 1 << 20), dtype=torch.float32, device=q.device,
                                         name="latent attention partials")
    for lo in range(0, b, step):
        hi = min(b, lo + step)
        qp, op, pos = _lib.ptr(q[lo:hi]), _lib.ptr(out[lo:hi]), _lib.ptr(positions[lo:hi])
        table = _lib.ptr(block_table if seq is not None else block_table[lo:hi])
        sq = _lib.ptr(None if seq is None else seq[lo:hi])
        if group:
            rc = L.b200_attn_latent_decode(qp, _lib.ptr(cache), op, table, sq, pos, _lib.ptr(ws), hi - lo, block_table.shape[1], nb, bs, m.heads,
                                           m.c, m.cache_width, int(splits), _f(m.scale), _lib.ptr(_lib.status_word(q.device)), _lib.stream())
            _lib.check(rc, "attn_latent_decode")
            if splits > 1:
                rc = L.b200_attn_latent_merge(_lib.ptr(ws), op, hi - lo, m.heads, m.c, int(splits), f32, _lib.stream())
                _lib.check(rc, "attn_latent_merge")
        else:
            rc = L.b200_attn_latent_rows(qp, _lib.ptr(cache), op, table, sq, pos, _lib.ptr(ws), hi - lo, block_table.shape[1], bs, m.heads, m.c,
                                         m.cache_width, int(splits), _f(m.scale), f32, _lib.stream())
            _lib.check(rc, "attn_latent_rows", 2 if splits > 1 else 1)
    return out


def tiles_supported(m: LatentAttention) -> bool:
    return bool(_lib.lib().b200_attn_heads_prefill_supported(m.heads, m.d, m.r, m.v))


def gather(cache: torch.Tensor, m: LatentAttention, block_table, seq, kv_len, kv_start, total: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Contexts of several sequences, one after the other: latents [rows, c] and rotated key parts [rows, 64-column slabs].
    Rows are rounded up to 256 with zero rows, so that the expansion tiles evenly."""
    nb, bs, _ = cache.shape
    _lib.check_indices(block_table, 0, nb, 3)
    rows, key_ld = (total + 255) // 256 * 256, max(64, (m.r + 63) // 64 * 64)
    lat = torch.empty(rows, m.c, dtype=cache.dtype, device=cache.device)
    key = torch.empty(rows, key_ld, dtype=cache.dtype, device=cache.device)
    rc = _lib.lib().b200_latent_gather(_lib.ptr(cache), _lib.ptr(block_table), _lib.ptr(seq), _lib.ptr(kv_len), _lib.ptr(kv_start),
                                       kv_len.numel(), block_table.shape[1], bs, m.c, m.r, key_ld, _lib.ptr(lat), _lib.ptr(key), rows,
                                       _lib.stream())
    _lib.check(rc, "latent_gather")
    return lat, key


def attend_tiles(q: torch.Tensor, m: LatentAttention, lat: torch.Tensor, key: torch.Tensor, w_kv, q_start, q_len, kv_len, kv_start,
                 max_q_len: int, out: torch.Tensor) -> torch.Tensor:
    """Rows of several sequences' portions.  q [rows, >= heads (d + r)], rotated; ``lat`` / ``key`` from ``gather``; ``w_kv``
    (``PackedLinear``): rows per head [d | v] that expand a latent; ``out`` [rows, >= heads v] in place."""
    from . import gemm
    rows, per = lat.shape[0], m.d + m.v
    group = max(1, min(m.heads, EXPANDED_LIMIT // (rows * per)))
    L = _lib.lib()
    for h0 in range(0, m.heads, group):
        n = min(group, m.heads - h0)
        part = gemm.PackedLinear(w_kv.wfmt, w_kv.weight[h0 * per:(h0 + n) * per], None, n * per, m.c)
        kv = gemm.linear(lat, part)
        rc = L.b200_attn_heads_prefill(
            _lib.ptr(q), q.stride(0), _lib.ptr(kv), _lib.ptr(key), key.shape[1], _lib.ptr(out), out.stride(0), _lib.ptr(q_start),
            _lib.ptr(q_len), _lib.ptr(kv_len), _lib.ptr(kv_start), q_len.numel(), int(max_q_len), q.shape[0], rows, h0, n, m.d, m.r, m.v,
            _f(m.scale), _lib.ptr(_lib.status_word(out.device)), _lib.stream())
        _lib.check(rc, "attn_heads_prefill")
    return out
