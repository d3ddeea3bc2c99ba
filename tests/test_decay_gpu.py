"""Recurrences with one decay per head on the GPU: the delta rule and retention against the plain token-by-token statement, in
whole prompts, portions, single rows and mixed batches, with states carried from slot to slot and slots used again."""
import pytest
import torch

from deepseek_v4_2080ti_b200.models.reference_cpu import nunosun_ref as ref
from deepseek_v4_2080ti_b200.ops import decay
from deepseek_v4_2080ti_b200.ops.scan import Segments

pytestmark = pytest.mark.gpu
DEV = "cuda"
EPS = 1e-5
pad = lambda n: (n + 15) // 16 * 16


def segments(entries):
    """(length, slot) per entry -> Segments over neighbouring rows."""
    first, row_first, row_slot, at = [], [], [], 0
    for n, slot in entries:
        first.append(at)
        row_first += [at] * n
        row_slot += [slot] * n
        at += n
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    lens = [n for n, _ in entries]
    return Segments(i32(row_first), i32(row_slot), i32(first), i32(lens), i32([s for _, s in entries]), max(lens), min(lens))


class Mixer:
    """One mixer with its own plain statement; ``rows`` makes projections, ``run`` feeds entries (sequence, from, to, slot)."""
    slots = 5

    def __init__(self, kind, heads, groups, dim, vdim, dtype, rot=None, taps=4, seed=0, strong=False):
        self.kind, self.heads, self.groups, self.dim, self.vdim, self.dtype = kind, heads, groups, dim, vdim, dtype
        gen = self.gen = torch.Generator().manual_seed(seed)
        d, v = pad(dim), pad(vdim)
        self.d, self.v = d, v
        row = lambda x, n: torch.cat([x.float(), torch.zeros(n - x.numel())]).to(DEV)
        if kind == "retention":
            self.decay = 1.0 - 2.0 ** (-torch.linspace(0.1 if strong else 1.0, 9.0, heads, dtype=torch.float64))
            self.rot = dim if rot is None else rot
            f = 500.0 ** (-torch.arange(0, self.rot, 2, dtype=torch.float64) / max(self.rot, 1))
            self.m = decay.Retention(heads, dim, d, vdim, v, EPS, self.rot, f.to(DEV), self.decay.float().to(DEV), torch.log2(self.decay).float().to(DEV),
                                     torch.ones(v, device=DEV))
            self.parts = [("q", heads, dim, d), ("k", heads, dim, d), ("v", heads, vdim, v), ("g", heads, vdim, v)]
        else:
            self.a_log, self.dt = torch.randn(heads, generator=gen) * (2.0 if strong else 0.7), torch.randn(heads, generator=gen) - 2.0
            self.norm = 1 + 0.2 * torch.randn(vdim, generator=gen)
            self.conv = {n: torch.randn(h, x, taps, generator=gen) / taps ** 0.5 for n, h, x in (("q", groups, dim), ("k", groups, dim), ("v", heads, vdim))}
            w = []
            for n, p in (("q", d), ("k", d), ("v", v)):
                c = self.conv[n]
                full = torch.zeros(c.shape[0], p, taps)
                full[:, :c.shape[1]] = c
                w.append(full.reshape(-1, taps))
            self.m = decay.DeltaRule(heads, groups, dim, d, vdim, v, EPS, torch.cat(w).t().contiguous().to(DEV),
                                     (-torch.exp(self.a_log)).to(DEV), self.dt.to(DEV), row(self.norm, v))
            self.parts = [("q", groups, dim, d), ("k", groups, dim, d), ("v", heads, vdim, v), ("g", heads, vdim, v), ("a", 1, heads, heads), ("b", 1, heads, heads)]
            self.tail = torch.full((self.slots, max(taps - 1, 1), self.m.channels), 7.0, dtype=dtype, device=DEV)
        self.state = torch.full((self.slots, heads, d, v), 3.0, device=DEV)                  # left over from other sequences
        self.ldo = heads * v + 16

    def rows(self, t):
        """[T, columns] projections, padded columns zero."""
        out = []
        for _, h, real, p in self.parts:
            x = torch.zeros(t, h, p)
            x[:, :, :real] = torch.randn(t, h, real, generator=self.gen)
            out.append(x.view(t, -1))
        out = torch.cat(out, 1)
        full = torch.zeros(t, pad(out.shape[1]) + 8)
        full[:, :out.shape[1]] = out
        return full.to(self.dtype)

    def want(self, rows):
        """fp64 rows [T, heads, vdim] of a whole sequence."""
        x, at, t = {}, 0, rows.shape[0]
        for n, h, real, p in self.parts:
            x[n] = rows[:, at:at + h * p].double().view(t, h, p)[:, :, :real]
            at += h * p
        if self.kind == "retention":
            q, k = (ref.rotate_half(x[n], range(t), self.rot, 500.0) for n in ("q", "k"))
            o, _ = ref.retention_recurrence(q, k * self.dim ** -0.5, x["v"], self.decay)
            return ref.rms(o, EPS) * ref.silu(x["g"])
        y = {n: ref.silu(ref.causal_conv(x[n].reshape(t, -1), self.conv[n].double().reshape(-1, self.conv[n].shape[2]))).view(x[n].shape)
             for n in ("q", "k", "v")}
        if self.dtype == torch.bfloat16:                        # the convolution's results are stored in the activations' type
            y = {n: z.bfloat16().double() for n, z in y.items()}
        wide = lambda z: ref.unit(z).repeat_interleave(self.heads // self.groups, 1)
        ld = -torch.exp(self.a_log.double()) * ref.softplus(x["a"][:, 0] + self.dt.double())
        o, _ = ref.delta_recurrence(wide(y["q"]) * self.dim ** -0.5, wide(y["k"]), y["v"], ld, ref.sigmoid(x["b"][:, 0]))
        return ref.rms(o, EPS) * self.norm.double() * ref.silu(x["g"])

    def run(self, entries):
        """entries: (rows of the sequence, from, to, slot) -> outputs per entry [n, heads, vdim]."""
        seg = segments([(b - a, s) for _, a, b, s in entries])
        proj = torch.cat([r[a:b] for r, a, b, _ in entries]).to(DEV)
        pos = torch.cat([torch.arange(a, b, dtype=torch.int32) for _, a, b, _ in entries]).to(DEV)
        if self.kind == "retention":
            out = decay.retention(proj, self.m, self.state, seg, pos, self.ldo)
        else:
            out = decay.delta_rule(proj, self.m, self.state, self.tail, seg, pos, self.ldo)
        assert out[:, self.heads * self.v:].abs().max() == 0
        out = out[:, :self.heads * self.v].view(-1, self.heads, self.v)
        assert out[:, :, self.vdim:].abs().max() == 0 if self.v > self.vdim else True
        parts, at = [], 0
        for _, a, b, _ in entries:
            parts.append(out[at:at + b - a, :, :self.vdim].cpu().double())
            at += b - a
        return parts


def close(got, want, dtype):
    err = ((got - want).norm(dim=(1, 2)) / want.norm(dim=(1, 2)).clamp(min=1e-2)).max().item()
    assert err < (1.2e-2 if dtype == torch.bfloat16 else 3e-5), err


DTYPES = [torch.bfloat16, torch.float32]
SHAPES = [("delta", 4, 2, 32, 64), ("delta", 3, 3, 20, 36), ("delta", 6, 1, 128, 128), ("delta", 2, 2, 200, 80), ("delta", 12, 4, 64, 160),
          ("retention", 4, 4, 64, 32), ("retention", 3, 3, 36, 20), ("retention", 5, 5, 128, 144), ("retention", 2, 2, 240, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_prompts_and_portions(shape, dtype):
    m = Mixer(*shape, dtype)
    rows = m.rows(331)
    want = m.want(rows)
    close(m.run([(rows, 0, 331, 2)])[0], want, dtype)
    # cut anywhere, also into single rows and pairs; the slot is used again
    cuts = [0, 2, 3, 66, 68, 100, 101, 117, 245, 247, 310, 331]
    close(torch.cat([m.run([(rows, a, b, 2)])[0] for a, b in zip(cuts, cuts[1:])]), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [SHAPES[0], SHAPES[2], SHAPES[3], SHAPES[5], SHAPES[7]])
def test_decoding(shape, dtype):
    m = Mixer(*shape, dtype, seed=1)
    a, b = m.rows(60), m.rows(45)
    wa, wb = m.want(a), m.want(b)
    got = m.run([(a, 0, 20, 0), (b, 0, 5, 3)])
    for t in range(40):                                       # two sequences, one row each
        x = m.run([(b, 5 + t, 6 + t, 3), (a, 20 + t, 21 + t, 0)])
        got = [torch.cat([got[0], x[1]]), torch.cat([got[1], x[0]])]
    close(got[0], wa, dtype)
    close(got[1], wb, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["delta", "retention"])
def test_mixed_batches(kind, dtype):
    m = Mixer(kind, 4, 2 if kind == "delta" else 4, 48, 32, dtype, seed=2, **({"rot": 32} if kind == "retention" else {"taps": 3}))
    seqs = [m.rows(n) for n in (200, 150, 97, 64)]
    want = [m.want(s) for s in seqs]
    got = [[] for _ in seqs]
    steps = [[(0, 0, 70), (1, 0, 1)], [(1, 1, 3), (0, 70, 71), (2, 0, 40)], [(2, 40, 56), (3, 0, 64), (0, 71, 199), (1, 3, 4)],
             [(0, 199, 200), (1, 4, 130)], [(1, 130, 150), (2, 56, 97)]]
    for step in steps:
        for (i, *_), x in zip(step, m.run([(seqs[i], a, b, i + 1) for i, a, b in step])):
            got[i].append(x)
    for g, w in zip(got, want):
        close(torch.cat(g), w, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["delta", "retention"])
def test_strong_and_weak_decays(kind, dtype):
    """Heads that forget within a token beside heads that keep hundreds: no factor may overflow."""
    m = Mixer(kind, 6, 6, 32, 32, dtype, seed=3, strong=True)
    rows = m.rows(300)
    if kind == "delta":
        at = sum(h * p for _, h, _, p in m.parts[:4])
        rows[::7, at:at + 6] = 60.0                            # the step opens fully now and then
    close(m.run([(rows, 0, 300, 1)])[0], m.want(rows), dtype)


@pytest.mark.parametrize("taps", [1, 2, 7])
def test_convolution_taps(taps):
    m = Mixer("delta", 2, 1, 32, 16, torch.float32, taps=taps, seed=4)
    rows = m.rows(90)
    cuts = [0, 2, 4, 5, 6, 30, 31, 33, 90]
    close(torch.cat([m.run([(rows, a, b, 4)])[0] for a, b in zip(cuts, cuts[1:])]), m.want(rows), torch.float32)


@pytest.mark.parametrize("rot", [0, 2, 32])
def test_partial_rotation(rot):
    m = Mixer("retention", 2, 2, 40, 16, torch.float32, rot=rot, seed=5)
    rows = m.rows(70)
    close(torch.cat([m.run([(rows, a, b, 0)])[0] for a, b in ((0, 50), (50, 51), (51, 70))]), m.want(rows), torch.float32)


def test_a_first_write_is_read_back_far_away():
    """One strong key at the first token of a slow head, zero writes after it: the last rows read it out."""
    for kind in ("delta", "retention"):
        m = Mixer(kind, 2, 2, 32, 32, torch.bfloat16, seed=6, **({"rot": 0} if kind == "retention" else {}))
        n = 400
        rows = m.rows(n)
        hv = 2 * 2 * 32
        rows[1:, hv:hv + 64] = 0                               # values after the first are nothing
        if kind == "retention":
            rows[:, :64] = rows[0, 64:128]                     # every query asks for the first key
        else:
            m.a_log.fill_(-8.0)
            m.m.neg_a = (-torch.exp(m.a_log)).to(DEV)
        want = m.want(rows)
        got = torch.cat([m.run([(rows, a, b, 1)])[0] for a, b in ((0, 129), (129, n - 1), (n - 1, n))])
        assert want[-1].abs().max() > 1e-2
        close(got, want, torch.bfloat16)
