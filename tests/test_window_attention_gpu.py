"""Attention with a sliding window and a distance bias on the GPU: prompt tiles, single rows and the prologue against a dense
statement, with keys that stand out just inside and just outside the window, at page borders and at the bias table's steps."""
import math

import pytest
import torch

from deepseek_v4_2080ti_b200.models.reference_cpu import nunosun_ref as ref
from deepseek_v4_2080ti_b200.ops import winattn

pytestmark = pytest.mark.gpu
DEV = "cuda"


def mixer(heads, groups, dim, vdim, size, rows=16, reach=64, scale=None, seed=0):
    gen = torch.Generator().manual_seed(seed)
    d, v = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    rel = torch.randn(rows, heads, generator=gen)
    w = lambda n, pad: torch.cat([1 + 0.2 * torch.randn(n, generator=gen), torch.zeros(pad - n)]).to(DEV)
    m = winattn.WindowAttention(heads, groups, dim, d, vdim, v, dim ** -0.5 if scale is None else scale, size, 1e-5, w(dim, d), w(dim, d),
                                winattn.distance_bias(rel.to(DEV), size, reach))
    return m, rel.double()


def dense(q, k, v, m, rel, reach, pos):
    """q [n, H, d] at positions ``pos``; k [T, G, d], v [T, G, v] fp64 -> [n, H, v]."""
    back = pos[:, None] - torch.arange(k.shape[0])[None, :]
    table = torch.tensor([ref.bucket(i, rel.shape[0], reach) for i in range(k.shape[0])])
    hidden = (back < 0) | (back >= m.size)
    out = []
    for h in range(m.heads):
        g = h // (m.heads // m.groups)
        s = (q[:, h] @ k[:, g].t() * m.scale + rel[table[back.clamp(min=0)], h]).masked_fill(hidden, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


def paged(x, bs, table, pages):
    """[T, w] rows into the pages of ``table``."""
    out = torch.zeros(pages, bs, x.shape[1], dtype=x.dtype, device=DEV)
    for i, b in enumerate(table):
        part = x[i * bs:(i + 1) * bs]
        out[b, :part.shape[0]] = part
    return out


def sequences(m, lens, bs, dtype, seed, spike=None):
    """Random keys and values of several sequences in shuffled pages; ``spike``: distances at which a query's own key direction
    is planted, so that one key takes most of the weight."""
    gen = torch.Generator().manual_seed(seed)
    per = [(n + bs - 1) // bs for n in lens]
    order = (torch.randperm(sum(per), generator=gen) + 1).tolist()
    kc = torch.zeros(sum(per) + 1, bs, m.k_width, dtype=dtype, device=DEV)
    vc = torch.zeros(sum(per) + 1, bs, m.v_width, dtype=dtype, device=DEV)
    bt = torch.zeros(len(lens), max(per), dtype=torch.int32)
    seqs = []
    for i, n in enumerate(lens):
        q, k = torch.randn(n, m.heads, m.d, generator=gen), torch.randn(n, m.groups, m.d, generator=gen)
        v = torch.randn(n, m.groups, m.v, generator=gen)
        q[:, :, m.dim:], k[:, :, m.dim:], v[:, :, m.vdim:] = 0, 0, 0
        if spike:
            for p in range(n):
                at = p - spike[p % len(spike)]
                if at >= 0:
                    q[p] = 3.0 * k[at].repeat_interleave(m.heads // m.groups, 0)
        q, k, v = (x.to(dtype) for x in (q, k, v))
        table = order[:per[i]]
        order = order[per[i]:]
        bt[i, :per[i]] = torch.tensor(table, dtype=torch.int32)
        kc += paged(k.reshape(n, -1).to(DEV), bs, table, kc.shape[0])
        vc += paged(v.reshape(n, -1).to(DEV), bs, table, vc.shape[0])
        seqs.append((q, k, v))
    return seqs, kc, vc, bt.to(DEV)


def err(a, b):
    return ((a.double().cpu() - b).norm(dim=-1) / b.norm(dim=-1).clamp(min=1e-3)).max().item()


SHAPES = [(4, 2, 64, 32, 40), (3, 3, 16, 16, 1), (6, 2, 128, 128, 300), (2, 1, 48, 80, 128), (5, 5, 32, 96, 129), (2, 2, 192, 160, 77),
          (8, 1, 80, 64, 1000), (32, 1, 64, 64, 200)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [16, 64])
def test_prompt_tiles(shape, bs):
    heads, groups, dim, vdim, size = shape
    m, rel = mixer(heads, groups, dim, vdim, size)
    assert winattn.tiles_supported(m, bs)
    lens, new = [700, 17, 391, 64], [700, 17, 140, 33]                    # whole prompts and portions behind a context
    seqs, kc, vc, bt = sequences(m, lens, bs, torch.bfloat16, 1, [0, max(size - 1, 0), size, size // 2])
    q = torch.cat([s[0][n - a:] for s, n, a in zip(seqs, lens, new)]).to(DEV).contiguous()
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    start = [sum(new[:i]) for i in range(len(new))]
    out = torch.full((q.shape[0], heads * m.v), float("nan"), dtype=torch.bfloat16, device=DEV)
    winattn.prefill(q, m, kc, vc, bt, i32(start), i32(new), i32(lens), max(new), out)
    winattn._lib.check_status()
    for (qs, k, v), n, a, s in zip(seqs, lens, new, start):
        want = dense(qs[n - a:].double(), k.double(), v.double(), m, rel, 64, torch.arange(n - a, n))
        assert err(out[s:s + a].view(a, heads, m.v), want) < 2e-2


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", SHAPES + [(3, 1, 320, 400, 50), (34, 2, 32, 32, 90)])
@pytest.mark.parametrize("splits", [None, 1, 3])
def test_single_rows(shape, dtype, splits):
    heads, groups, dim, vdim, size = shape
    m, rel = mixer(heads, groups, dim, vdim, size)
    bs, lens = 32, [1, 2, 40, 41, 129, 300, 301, 1100]
    seqs, kc, vc, bt = sequences(m, lens, bs, dtype, 2, [max(size - 1, 0)])
    q = torch.stack([s[0][-1] for s in seqs]).to(DEV).contiguous()
    pos = torch.tensor([n - 1 for n in lens], dtype=torch.int32, device=DEV)
    out = torch.empty(len(lens), heads * m.v, dtype=dtype, device=DEV)
    winattn.rows(q, m, kc, vc, bt, pos, max(lens), out, splits=splits)
    tol = 2e-2 if dtype == torch.bfloat16 else 5e-6
    for i, ((qs, k, v), n) in enumerate(zip(seqs, lens)):
        want = dense(qs[-1:].double(), k.double(), v.double(), m, rel, 64, torch.tensor([n - 1]))
        assert err(out[i].view(1, heads, m.v), want) < tol
    # the same rows through table rows given by name, in another order
    order = torch.tensor([5, 0, 7, 3], device=DEV)
    again = torch.empty(4, heads * m.v, dtype=dtype, device=DEV)
    winattn.rows(q[order].contiguous(), m, kc, vc, bt, pos[order].contiguous(), max(lens), again, seq=order.int(), splits=splits)
    assert torch.equal(again, out[order])


def test_pages_in_front_of_the_window_are_not_needed():
    m, rel = mixer(4, 2, 64, 64, 50)
    bs, lens, new = 16, [400], [100]
    seqs, kc, vc, bt = sequences(m, lens, bs, torch.bfloat16, 3)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    q = seqs[0][0][300:].to(DEV).contiguous()
    run = lambda table: (winattn.prefill(q, m, kc, vc, table, i32([0]), i32(new), i32(lens), 100, torch.empty(100, 256, dtype=torch.bfloat16, device=DEV)),
                         winattn.rows(q[-1:].contiguous(), m, kc, vc, table, i32([399]), 400, torch.empty(1, 256, dtype=torch.bfloat16, device=DEV)))
    a, b = run(bt)
    gone = bt.clone()
    gone[0, :(300 - 49) // bs] = 0
    c, d = run(gone)
    assert torch.equal(a, c) and torch.equal(b, d)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_prologue(dtype):
    m, _ = mixer(4, 2, 40, 24, 10)
    gen = torch.Generator().manual_seed(5)
    t, bs = 9, 16
    proj = torch.zeros(t, m.q_width + m.k_width + m.v_width + 48)
    parts = {}
    at = 0
    for n, h, real, pad in (("q", 4, 40, m.d), ("k", 2, 40, m.d), ("v", 2, 24, m.v)):
        parts[n] = torch.randn(t, h, real, generator=gen).to(dtype)
        proj[:, at:at + h * pad].view(t, h, pad)[:, :, :real] = parts[n].float()
        at += h * pad
    kc, vc = (torch.zeros(3, bs, w, dtype=dtype, device=DEV) for w in (m.k_width, m.v_width))
    slots = torch.tensor([17, 18, 40, 41, 20, 21, 22, 47, 16], dtype=torch.int32, device=DEV)
    q = winattn.head_prep(proj.to(DEV, dtype), m, torch.arange(t, dtype=torch.int32, device=DEV), slots, kc, vc)
    tol = 1e-2 if dtype == torch.bfloat16 else 1e-6
    for got, part, w in ((q, "q", m.q_w), (kc.view(-1, 2, m.d)[slots.long()], "k", m.k_w)):
        want = ref.rms(parts[part].double(), m.eps) * w[:40].double().cpu()
        assert err(got[:, :, :40], want) < tol and got[:, :, 40:].abs().max() == 0
    assert torch.equal(vc.view(-1, 2, m.v)[slots.long()][:, :, :24].cpu(), parts["v"])
