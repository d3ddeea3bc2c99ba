"""Convolution and selective-scan kernels against the plain statement: every state count the kernel has a form for, portions
of one sequence against the whole, several sequences in one launch, time slices, and slots that held something else."""
import pytest
import torch

from deepseek_v4_2080ti_b200.models.reference_cpu import zigasun_ref as ref

pytestmark = pytest.mark.gpu
DT = {torch.bfloat16: 1e-2, torch.float32: 3e-6}
BOTH = pytest.mark.parametrize("dtype", list(DT))


def _mods():
    from deepseek_v4_2080ti_b200.ops import _lib, scan
    return _lib, scan


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-30))


def _segments(entries):
    """entries: (slot, length) in row order."""
    _, sc = _mods()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32).cuda()
    first, at = [], 0
    for _, n in entries:
        first.append(at)
        at += n
    rows = [(f, s) for f, (s, n) in zip(first, entries) for _ in range(n)]
    lens = [n for _, n in entries]
    return sc.Segments(i32([f for f, _ in rows]), i32([s for _, s in rows]), i32(first), i32(lens), i32([s for s, _ in entries]),
                       max(lens), min(lens))


class Seq:
    """Inputs of one sequence of the recurrence and the statement's answer."""

    def __init__(self, n, c, states, dtype, seed, slow=False):
        gen = torch.Generator().manual_seed(seed)
        r = lambda *s: torch.randn(*s, generator=gen)
        self.x, self.z = r(n, c).to(dtype), r(n, c).to(dtype)
        self.b, self.c = r(n, states).to(dtype), r(n, states).to(dtype)
        self.dt = (-7.0 if slow else -2.0) + 1.5 * r(n, c)
        if slow:                                        # the first token is worth hundreds of the others
            self.dt[0] = 6.0
            self.x[0] = 3.0


class Rec:
    def __init__(self, c, states, dtype, slots=5, taps=4, seed=0):
        _, sc = _mods()
        gen = torch.Generator().manual_seed(100 + seed)
        self.C, self.N, self.dtype, self.taps = c, states, dtype, taps
        self.a_log = torch.log(torch.arange(1, states + 1).float()).expand(c, states) * 0.5 - 1.0 + 0.3 * torch.randn(c, states, generator=gen)
        self.bias, self.d = 0.5 * torch.randn(c, generator=gen), torch.randn(c, generator=gen)
        self.a = sc.scan_decay(self.a_log, dtype).cuda()
        # whatever an earlier request left behind must not show
        self.state = torch.full((slots, c, states), float("nan")).cuda()
        self.tail = torch.full((slots, max(taps - 1, 1), c), float("nan"), dtype=dtype).cuda()
        self.n8 = (states + 7) // 8 * 8
        self.w = torch.randn(taps, c, generator=gen)
        self.cb = torch.randn(c, generator=gen)

    def want(self, s):
        d = lambda t: t.double()
        y, st = ref.selective_scan(d(s.x), ref.softplus(d(s.dt) + d(self.bias)), -torch.exp(d(self.a_log)), d(s.b), d(s.c), d(self.d))
        return y * ref.silu(d(s.z)), st

    def run(self, parts, slices=None):
        """parts: (slot, Seq, lo, hi) -> output rows per part."""
        _, sc = _mods()
        cat = lambda f: torch.cat([f(s)[lo:hi] for _, s, lo, hi in parts]).cuda()
        rows = sum(hi - lo for _, _, lo, hi in parts)
        bc = torch.zeros(rows, 8 + 2 * self.n8, dtype=self.dtype).cuda()
        bc[:, 8:8 + self.N], bc[:, 8 + self.n8:8 + self.n8 + self.N] = cat(lambda s: s.b), cat(lambda s: s.c)
        bc[:, :8] = 77.0
        x = cat(lambda s: s.x)
        xz = torch.cat([x, cat(lambda s: s.z)], 1)
        pos = torch.tensor([p for _, _, lo, hi in parts for p in range(lo, hi)], dtype=torch.int32).cuda()
        seg = _segments([(slot, hi - lo) for slot, _, lo, hi in parts])
        out = sc.selective_scan(x, cat(lambda s: s.dt), bc, 8, 8 + self.n8, xz[:, self.C:], self.a, self.bias.cuda(), self.d.cuda(),
                                self.state, seg, pos, xz[:, :self.C], self.tail, slices=slices)
        return list(out.split([hi - lo for _, _, lo, hi in parts]))

    def conv(self, parts):
        _, sc = _mods()
        x = torch.cat([s.x[lo:hi] for _, s, lo, hi in parts]).cuda()
        pos = torch.tensor([p for _, _, lo, hi in parts for p in range(lo, hi)], dtype=torch.int32).cuda()
        seg = _segments([(slot, hi - lo) for slot, _, lo, hi in parts])
        return list(sc.conv_rows(x, self.w.cuda(), self.cb.cuda(), self.tail, seg, pos).split([hi - lo for _, _, lo, hi in parts]))


@BOTH
@pytest.mark.parametrize("states", [1, 3, 4, 7, 8, 13, 16, 20, 24, 32, 40, 64, 100, 128, 200, 256])
def test_state_counts(states, dtype):
    c = Rec(48 if states > 64 else 88, states, dtype, seed=states)
    s = Seq(75, c.C, states, dtype, states)
    want, st = c.want(s)
    got = c.run([(2, s, 0, 75)])[0]
    assert _rel(got, want) < DT[dtype] and _rel(c.state[2], st) < (1e-5 if dtype == torch.float32 else 2e-4)
    assert torch.isnan(c.state[[0, 1, 3, 4]]).all()
    # one more token from the kept state
    s2 = Seq(76, c.C, states, dtype, states)
    for f in ("x", "z", "b", "c", "dt"):
        getattr(s2, f)[:75] = getattr(s, f)
    want, st = c.want(s2)
    got = c.run([(2, s2, 75, 76)])[0]
    assert _rel(got, want[75:]) < DT[dtype] and _rel(c.state[2], st) < (1e-5 if dtype == torch.float32 else 2e-4)


@BOTH
@pytest.mark.parametrize("cuts", [[1] * 40, [2] * 20, [3, 1, 36], [31, 9], [32, 8], [33, 7], [5, 5, 30], [39, 1]])
def test_portions_of_one_sequence(cuts, dtype):
    """The same outputs, states and convolution inputs however the sequence is cut."""
    c = Rec(72, 20, dtype)
    s = Seq(40, 72, 20, dtype, 5)
    want, st = c.want(s)
    conv_want = ref.silu(ref.causal_conv(s.x.double(), c.w.double().t(), c.cb.double()))
    at, got, conv = 0, [], []
    for n in cuts:
        conv += c.conv([(1, s, at, at + n)])
        got += c.run([(1, s, at, at + n)])
        at += n
    assert _rel(torch.cat(got), want) < DT[dtype] and _rel(c.state[1], st) < (1e-5 if dtype == torch.float32 else 2e-4)
    assert _rel(torch.cat(conv), conv_want) < (5e-3 if dtype == torch.bfloat16 else 1e-6)
    assert torch.equal(c.tail[1].cpu(), s.x[37:])


@BOTH
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_convolution_lengths(taps, dtype):
    c = Rec(40, 4, dtype, taps=taps)
    s = Seq(30, 40, 4, dtype, taps)
    want = ref.silu(ref.causal_conv(s.x.double(), c.w.double().t(), c.cb.double()))
    for cuts in ([30], [1] * 30, [2, 3, 1, 24]):
        at, got = 0, []
        for n in cuts:
            got += c.conv([(0, s, at, at + n)])
            c.run([(0, s, at, at + n)])
            at += n
        assert _rel(torch.cat(got), want) < (5e-3 if dtype == torch.bfloat16 else 1e-6), cuts


@BOTH
def test_unequal_sequences_in_one_launch(dtype):
    """Portions of several sequences beside single tokens of others, each equal to the sequence alone."""
    c = Rec(80, 16, dtype)
    seqs = [Seq(n, 80, 16, dtype, 10 + n) for n in (90, 3, 50, 1, 7)]
    wants = [c.want(s) for s in seqs]
    plan = [[(0, 0, 40), (3, 0, 1), (2, 0, 49)], [(1, 0, 2), (0, 40, 41), (2, 49, 50), (4, 0, 5)],
            [(4, 5, 6), (0, 41, 90), (1, 2, 3)], [(4, 6, 7)]]
    rows = {i: [] for i in range(5)}
    for step in plan:
        parts = [(4 - i, seqs[i], lo, hi) for i, lo, hi in step]
        for (i, _, _), o in zip(step, c.run(parts)):
            rows[i].append(o)
    for i, (want, st) in enumerate(wants):
        assert _rel(torch.cat(rows[i]), want) < DT[dtype], i
        assert _rel(c.state[4 - i], st) < (1e-5 if dtype == torch.float32 else 2e-4), i


@BOTH
@pytest.mark.parametrize("slices", [1, 2, 3, 8])
def test_time_slices(slices, dtype):
    """Cutting a long sequence over blocks composes the same states, from zero and from a kept state, beside a short one."""
    c = Rec(32, 12, dtype)
    s, t = Seq(700, 32, 12, dtype, 3), Seq(70, 32, 12, dtype, 4)
    (want, st), (want_t, st_t) = c.want(s), c.want(t)
    got = [c.run([(0, s, 0, 300), (1, t, 0, 64)], slices), c.run([(1, t, 64, 70), (0, s, 300, 700)], slices)]
    assert _rel(torch.cat([got[0][0], got[1][1]]), want) < DT[dtype]
    assert _rel(torch.cat([got[0][1], got[1][0]]), want_t) < DT[dtype]
    tol = 1e-5 if dtype == torch.float32 else 2e-4
    assert _rel(c.state[0], st) < tol and _rel(c.state[1], st_t) < tol


@BOTH
def test_a_first_token_that_matters_for_hundreds(dtype):
    """Slow decays and one loud first token: a state that is lost or started again anywhere shows in every later row."""
    c = Rec(64, 16, dtype)
    c.a_log -= 4.0
    _, sc = _mods()
    c.a = sc.scan_decay(c.a_log, dtype).cuda()
    s = Seq(420, 64, 16, dtype, 6, slow=True)
    want, st = c.want(s)
    lost = Seq(420, 64, 16, dtype, 6, slow=True)
    lost.x[0] = 0.0
    assert _rel(c.want(lost)[0][300:], want[300:]) > 0.3
    for cuts, slices in (([420], 4), ([33] * 12 + [24], 1), ([100, 1, 1, 318], 2)):
        at, got = 0, []
        for n in cuts:
            got += c.run([(3, s, at, at + n)], slices)
            at += n
        assert _rel(torch.cat(got), want) < DT[dtype]


def test_extreme_step_sizes():
    """Step sizes from the far tails of the softplus keep their digits in both forms of the kernel."""
    for dtype in DT:
        c = Rec(32, 8, dtype)
        s = Seq(40, 32, 8, dtype, 9)
        s.dt = torch.linspace(-20, 12, 40)[:, None].expand(40, 32).contiguous()
        c.bias.zero_()
        c.d.zero_()
        want, _ = c.want(s)
        assert _rel(c.run([(0, s, 0, 40)])[0], want) < DT[dtype]
        # tiny steps alone: y is proportional to them, so their relative accuracy is what is left
        s.dt = torch.full((40, 32), -15.0)
        want, _ = c.want(s)
        assert _rel(c.run([(0, s, 0, 40)])[0], want) < DT[dtype]
