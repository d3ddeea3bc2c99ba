"""Gated linear attention kernels against the plain statement: prompts in chunks, portions, single rows, several sequences in one
launch, decays from none to all in one token, kept first tokens, and slots that held something else."""
import pytest
import torch

from deepseek_v4_2080ti_b200.models.reference_cpu import kemirax_ref as ref

pytestmark = pytest.mark.gpu
DT = {torch.bfloat16: 6e-3, torch.float32: 5e-6}
BOTH = pytest.mark.parametrize("dtype", list(DT))
SIZES = [(2, 10, 14, 5, 16.0), (3, 48, 32, 16, 16.0), (1, 128, 128, 8, 4.0), (2, 70, 200, 40, 1.0), (1, 200, 24, 16, 0.5), (2, 300, 16, 16, 16.0)]
ALL = pytest.mark.parametrize("size", SIZES)          # heads, dim, vdim, rank, tau


def _mods():
    from deepseek_v4_2080ti_b200.ops import _lib, gla
    return _lib, gla


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-30))


def _pad(n):
    return (n + 15) // 16 * 16


def _segments(entries):
    """entries: (slot, length) in row order."""
    from deepseek_v4_2080ti_b200.ops.scan import Segments
    i32 = lambda v: torch.tensor(v, dtype=torch.int32).cuda()
    first, at = [], 0
    for _, n in entries:
        first.append(at)
        at += n
    rows = [(f, s) for f, (s, n) in zip(first, entries) for _ in range(n)]
    lens = [n for _, n in entries]
    return Segments(i32([f for f, _ in rows]), i32([s for _, s in rows]), i32(first), i32(lens), i32([s for s, _ in entries]), max(lens), min(lens))


class Rec:
    """One mixer with state slots; sequences are the projection's columns."""

    def __init__(self, size, dtype, slots=5, seed=0, bias=None):
        _, gla = _mods()
        self.heads, self.dim, self.vdim, rank, self.tau = size
        self.dtype, self.d, self.v, self.rank = dtype, _pad(self.dim), _pad(self.vdim), _pad(rank)
        gen = torch.Generator().manual_seed(seed + self.dim)
        h = self.heads
        self.w2 = torch.zeros(h, self.d, self.rank)
        self.w2[:, :self.dim, :rank] = 1.5 * torch.randn(h, self.dim, rank, generator=gen) / rank ** 0.5
        self.w2 = self.w2.to(dtype)
        self.b2 = torch.zeros(h, self.d)
        self.b2[:, :self.dim] = 2.0 + 2.0 * torch.randn(h, self.dim, generator=gen) if bias is None else bias
        self.nw = torch.zeros(self.v)
        self.nw[:self.vdim] = 1 + 0.3 * torch.randn(self.vdim, generator=gen)
        self.m = gla.GatedLinear(h, self.dim, self.d, self.vdim, self.v, self.tau, 1e-4, self.rank, self.w2.view(-1, self.rank).cuda().contiguous(),
                                 self.b2.view(-1).cuda(), self.nw.cuda())
        self.state = torch.full((slots, h, self.d, self.v), float("nan")).cuda()       # whatever was there must not show
        self.rank_real = rank

    def seq(self, n, seed):
        gen = torch.Generator().manual_seed(seed)
        oq, ok, ov, og, oa = self.m.offsets
        p = torch.zeros(n, oa + self.rank + 16)
        r = lambda *s: torch.randn(*s, generator=gen)
        for off, real, pad in ((oq, self.dim, self.d), (ok, self.dim, self.d), (ov, self.vdim, self.v), (og, self.vdim, self.v)):
            p[:, off:off + self.heads * pad].view(n, self.heads, pad)[:, :, :real] = r(n, self.heads, real)
        p[:, oa:oa + self.rank_real] = r(n, self.rank_real)
        p[:, -16:] = 50.0
        return p.to(self.dtype)

    def want(self, p):
        n, h = p.shape[0], self.heads
        oq, ok, ov, og, oa = self.m.offsets
        x = p.double()
        part = lambda off, real, pad: x[:, off:off + h * pad].view(n, h, pad)[:, :, :real]
        z = x[:, oa:oa + self.rank] @ self.w2.view(-1, self.rank).double().t() + self.b2.view(-1).double()
        la = (ref.log_sigmoid(z) / self.tau).view(n, h, self.d)[:, :, :self.dim]
        o, s = ref.gated_recurrence(part(oq, self.dim, self.d) * self.dim ** -0.5, part(ok, self.dim, self.d), part(ov, self.vdim, self.v), la)
        g = part(og, self.vdim, self.v)
        return ref.rms(o, 1e-4) * self.nw[:self.vdim].double() * g * ref.sigmoid(g), s

    def run(self, parts):
        """parts: (slot, sequence, lo, hi); returns rows [*, heads, vdim] per part."""
        _, gla = _mods()
        proj = torch.cat([p[lo:hi] for _, p, lo, hi in parts]).cuda()
        pos = torch.cat([torch.arange(lo, hi, dtype=torch.int32) for _, _, lo, hi in parts]).cuda()
        ldo = self.heads * self.v + 16
        out = gla.recurrence(proj, self.m, self.state, _segments([(s, hi - lo) for s, _, lo, hi in parts]), pos, ldo)
        assert not out[:, self.heads * self.v:].any()
        y = out[:, :self.heads * self.v].view(-1, self.heads, self.v)
        assert not y[:, :, self.vdim:].any()
        res, at = [], 0
        for _, _, lo, hi in parts:
            res.append(y[at:at + hi - lo, :, :self.vdim].double().cpu())
            at += hi - lo
        return res

    def final(self, slot):
        return self.state[slot, :, :self.dim, :self.vdim]


@BOTH
@ALL
@pytest.mark.parametrize("n", [1, 2, 15, 16, 17, 63, 64, 65, 200])
def test_whole_prompts(dtype, size, n):
    r = Rec(size, dtype)
    p = r.seq(n, n)
    want, s = r.want(p)
    got, = r.run([(3, p, 0, n)])
    assert _rel(got, want) < DT[dtype] and _rel(r.final(3), s) < DT[dtype]
    assert torch.isnan(r.state[[0, 1, 2, 4]]).all()


@BOTH
@ALL
def test_portions_and_single_rows_continue_the_state(dtype, size):
    r = Rec(size, dtype)
    p = r.seq(170, 7)
    want, s = r.want(p)
    for cuts in ([1] * 8 + [30, 2, 64, 1, 65], [100, 16, 15, 39], [64, 64, 42], [3] * 6 + [152]):
        at, rows = 0, []
        for n in cuts:
            rows += r.run([(1, p, at, at + n)])
            at += n
        assert at == 170 and _rel(torch.cat(rows), want) < DT[dtype] and _rel(r.final(1), s) < DT[dtype], cuts


@BOTH
@ALL
def test_unequal_sequences_in_one_launch(dtype, size):
    r = Rec(size, dtype)
    ps = {s: r.seq(n, 20 + s) for s, n in ((0, 130), (2, 90), (3, 40), (4, 3))}
    want = {s: r.want(p) for s, p in ps.items()}
    rows = {s: [] for s in ps}
    for batch in ([(0, 0, 50), (3, 0, 1), (2, 0, 17)], [(3, 1, 2), (0, 50, 51), (4, 0, 2), (2, 17, 81)], [(2, 81, 82), (0, 51, 52), (4, 2, 3), (3, 2, 3)],
                  [(0, 52, 130), (2, 82, 90), (3, 3, 40)]):
        for (s, _, _), y in zip(batch, r.run([(s, ps[s], lo, hi) for s, lo, hi in batch])):
            rows[s].append(y)
    for s in ps:
        assert _rel(torch.cat(rows[s]), want[s][0]) < DT[dtype] and _rel(r.final(s), want[s][1]) < DT[dtype], s
    # a slot used again starts from nothing
    p = r.seq(70, 99)
    got, = r.run([(0, p, 0, 70)])
    assert _rel(got, r.want(p)[0]) < DT[dtype]


@BOTH
@pytest.mark.parametrize("bias", [-300.0, -40.0, -8.0, 30.0])
def test_decays_from_all_to_nothing(dtype, bias):
    """Channels that forget everything within one row, and channels that never do; no factor overflows on the way."""
    size = (2, 48, 32, 16, 1.0)
    r = Rec(size, dtype, bias=bias)
    r.b2[:, ::3] = 30.0 if bias < 0 else -300.0                # both kinds side by side
    r.b2[:, r.dim:] = 0
    r.m.b2.copy_(r.b2.view(-1))
    p = r.seq(150, 3)
    want, s = r.want(p)
    for cuts in ([150], [64, 1, 1, 84], [1] * 5 + [145]):
        at, rows = 0, []
        for n in cuts:
            rows += r.run([(2, p, at, at + n)])
            at += n
        got = torch.cat(rows)
        assert bool(torch.isfinite(got).all()) and _rel(got, want) < DT[dtype] and _rel(r.final(2), s) < DT[dtype]


@BOTH
def test_the_first_token_is_kept_for_long(dtype):
    """Slow decays and one loud key at the start: hundreds of rows later the output is still mostly its value."""
    r = Rec((1, 64, 32, 16, 16.0), dtype, bias=12.0)
    r.m.w2.zero_()
    r.w2 = torch.zeros_like(r.w2)
    p = r.seq(520, 4)
    oq, ok, ov, _, _ = r.m.offsets
    p[0, ok:ok + 64] = 12.0
    p[:, oq:oq + 64] = p[:, oq:oq + 64].abs()
    want, s = r.want(p)
    other = p.clone()
    other[0, ov:ov + 32] = -other[0, ov:ov + 32]
    assert _rel(r.want(other)[0][500:], want[500:]) > 0.5                # it shows
    for cuts in ([520], [64, 65, 391], [400] + [1] * 120):
        at, rows = 0, []
        for n in cuts:
            rows += r.run([(0, p, at, at + n)])
            at += n
        # five hundred decays of nearly one: their own rounding in fp32 adds up
        tol = max(DT[dtype], 4e-5)
        assert _rel(torch.cat(rows)[500:], want[500:]) < tol and _rel(r.final(0), s) < tol
