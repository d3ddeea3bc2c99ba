"""Differential-attention kernels against the plain statement (``models/reference_cpu/zigasun_ref.py``): prologue, prompt tiles
and single rows, in sizes that are multiples of nothing, with keys made to stand out at the places where a kernel's tiles,
pages and slices meet."""
import pytest
import torch

from deepseek_v4_2080ti_b200.models.reference_cpu import zigasun_ref as ref

pytestmark = pytest.mark.gpu
DT = {torch.bfloat16: 2e-2, torch.float32: 5e-6}
BOTH = pytest.mark.parametrize("dtype", list(DT))
# heads, kv heads, dim, vdim
SHAPES = [(4, 2, 40, 56), (3, 1, 64, 128), (8, 1, 16, 16), (6, 3, 128, 64), (5, 5, 20, 200), (16, 1, 32, 96), (2, 2, 96, 256),
          (7, 1, 30, 40), (2, 1, 160, 48), (4, 1, 250, 130)]


def _mods():
    from deepseek_v4_2080ti_b200.ops import _lib, diffattn
    return _lib, diffattn


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-30))


def _gen(seed):
    return torch.Generator().manual_seed(seed)


class Attn:
    """One mixer with its cache filled for some sequences, and the statement's answer for any (sequence, position)."""

    def __init__(self, shape, dtype, lens, seed=0, block_size=64, diff=0.25, lam=0.8, scale=None, spike=None, pool=None):
        _, da = _mods()
        self.H, self.G, self.dim, self.vdim = shape
        pad = lambda n: (n + 15) // 16 * 16
        self.d, self.v, self.bs, self.dtype = pad(self.dim), pad(self.vdim), block_size, dtype
        self.m = da.DiffAttention(self.H, self.G, self.dim, self.d, self.vdim, self.v, scale or self.dim ** -0.5, lam, diff, 1e-4,
                                  torch.ones(self.d).cuda(), torch.ones(self.d).cuda())
        gen = _gen(seed)
        self.q, self.k, self.val, self.gate = [], [], [], []
        for i, n in enumerate(lens):
            q, k = torch.randn(n, self.H, 2, self.dim, generator=gen), torch.randn(n, self.G, 2, self.dim, generator=gen)
            if spike:
                spike(i, q, k)
            self.q.append(q.to(dtype))
            self.k.append(k.to(dtype))
            self.val.append(torch.randn(n, self.G, self.vdim, generator=gen).to(dtype))
            self.gate.append(torch.randn(n, self.H, generator=gen).to(dtype))
        need = [(n + block_size - 1) // block_size for n in lens]
        order = (torch.randperm(sum(need), generator=gen) + 1).tolist()
        nb = sum(need) + 1
        # pages hold large finite values wherever no token of a sequence lies
        self.kc = torch.full((nb, block_size, self.G * 2 * self.d), 50.0, dtype=dtype)
        self.vc = torch.full((nb, block_size, self.G * self.v), -70.0, dtype=dtype)
        self.kc[0], self.vc[0] = 0, 0
        self.bt = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
        for i, n in enumerate(lens):
            for b in range(need[i]):
                page = order.pop()
                self.bt[i, b] = page
                lo, hi = b * block_size, min(n, (b + 1) * block_size)
                kp, vp = torch.zeros(hi - lo, self.G, 2, self.d), torch.zeros(hi - lo, self.G, self.v)
                kp[..., :self.dim], vp[..., :self.vdim] = self.k[i][lo:hi], self.val[i][lo:hi]
                self.kc[page, :hi - lo], self.vc[page, :hi - lo] = kp.reshape(hi - lo, -1).to(dtype), vp.reshape(hi - lo, -1).to(dtype)
        self.kc, self.vc, self.bt = self.kc.cuda(), self.vc.cuda(), self.bt.cuda()

    def padded_q(self, parts):
        q = torch.cat(parts)
        out = torch.zeros(q.shape[0], self.H, 2, self.d, dtype=self.dtype)
        out[..., :self.dim] = q
        return out.cuda()

    def want(self, i):
        """[n, H, vdim] fp64, gated."""
        q, k, v = (t.double() for t in (self.q[i], self.k[i], self.val[i]))
        per = self.H // self.G
        out = []
        for h in range(self.H):
            a1, a2 = (ref.softmax_attention(q[:, h, m], k[:, h // per, m], v[:, h // per], self.m.scale) for m in (0, 1))
            out.append(ref.difference_of_maps(a1, a2, torch.tensor(self.m.lam, dtype=torch.float64), self.m.diff, self.m.eps))
        return torch.stack(out, 1) * torch.sigmoid(self.gate[i].double())[:, :, None]

    def rows(self, picks, splits=None, via_seq=True):
        """Row kernel for (sequence, position) picks -> [B, H, vdim]."""
        _, da = _mods()
        q = self.padded_q([self.q[i][p:p + 1] for i, p in picks])
        gate = torch.cat([self.gate[i][p:p + 1] for i, p in picks]).cuda()
        pos = torch.tensor([p for _, p in picks], dtype=torch.int32).cuda()
        out = torch.full((len(picks), self.H * self.v), 9.0, dtype=self.dtype).cuda()
        seq = torch.tensor([i for i, _ in picks], dtype=torch.int32).cuda()
        da.rows(q, self.m, self.kc, self.vc, gate, self.bt if via_seq else self.bt[seq.long()].contiguous(), pos,
                max(p for _, p in picks) + 1, out, seq=seq if via_seq else None, splits=splits)
        return self.check_pads(out)

    def check_pads(self, out):
        o = out.view(-1, self.H, self.v)
        assert not o[..., self.vdim:].any()
        return o[..., :self.vdim]

    def tiles(self, parts):
        """Tile kernel for portions (sequence, first position, end) -> list of [n, H, vdim]."""
        lib, da = _mods()
        i32 = lambda v: torch.tensor(v, dtype=torch.int32).cuda()
        q = self.padded_q([self.q[i][a:b] for i, a, b in parts])
        gate = torch.cat([self.gate[i][a:b] for i, a, b in parts]).cuda()
        lens = [b - a for _, a, b in parts]
        start = [sum(lens[:j]) for j in range(len(lens))]
        out = torch.full((sum(lens), self.H * self.v), 9.0, dtype=self.dtype).cuda()
        da.prefill(q, self.m, self.kc, self.vc, gate, self.bt, i32(start), i32(lens), i32([b for _, _, b in parts]), max(lens), out,
                   seq=i32([i for i, _, _ in parts]))
        lib.check_status()
        o = self.check_pads(out)
        return [o[s:s + n] for s, n in zip(start, lens)]


@BOTH
@pytest.mark.parametrize("shape", SHAPES)
def test_single_rows(shape, dtype):
    a = Attn(shape, dtype, [150, 33, 1], seed=sum(shape))
    picks = [(0, 149), (1, 32), (2, 0), (0, 0), (0, 63), (0, 64), (0, 15), (0, 16), (1, 1), (0, 127), (0, 128)]
    want = torch.stack([a.want(i)[p] for i, p in picks])
    for splits in (None, 1, 2, 7):
        got = a.rows(picks, splits)
        assert max(_rel(g, w) for g, w in zip(got, want)) < 3 * DT[dtype], splits
    assert _rel(a.rows(picks, via_seq=False), want) < DT[dtype]


@pytest.mark.parametrize("shape", SHAPES)
def test_prompt_tiles(shape):
    lib, da = _mods()
    a = Attn(shape, torch.bfloat16, [300, 130, 17], seed=1 + sum(shape))
    assert da.tiles_supported(a.m, 64)
    parts = [(0, 0, 300), (1, 100, 130), (2, 0, 17)]
    for got, (i, lo, hi) in zip(a.tiles(parts), parts):
        assert _rel(got, a.want(i)[lo:hi]) < DT[torch.bfloat16]


@pytest.mark.parametrize("block_size", [16, 32, 128])
def test_other_page_sizes(block_size):
    a = Attn((4, 2, 40, 56), torch.bfloat16, [200, 61], seed=5, block_size=block_size)
    w = a.want(0)
    assert _rel(a.tiles([(0, 70, 200)])[0], w[70:]) < DT[torch.bfloat16]
    assert _rel(a.rows([(0, 199), (1, 60)]), torch.stack([w[199], a.want(1)[60]])) < DT[torch.bfloat16]


def _one_key(where, who, gain=9.0):
    """Queries from position ``who`` on point at key ``where`` in both maps: its score stands far above all others."""
    def spike(i, q, k):
        n = q.shape[0]
        if i == 0 and n > where:
            per = q.shape[1] // k.shape[1]
            for h in range(q.shape[1]):
                for m in (0, 1):
                    # in the second map another key: the difference then shows both
                    at = where if m == 0 else max(where - 1, 0)
                    d = k[at, h // per, m] / k[at, h // per, m].norm()
                    k[at, h // per, m] = d * k.shape[-1] ** 0.5
                    q[who:, h, m] = 0.1 * q[who:, h, m] + d * gain
    return spike


@BOTH
@pytest.mark.parametrize("where", [0, 1, 15, 16, 63, 64, 127, 128, 129, 255, 256, 300, 511])
def test_one_far_key_among_hundreds(where, dtype):
    """A key that carries nearly all the weight, at tile, page and slice borders, seen from far away; leaving it out or
    reading its neighbour changes the answer completely."""
    a = Attn((4, 2, 48, 64), dtype, [600, 40], seed=where, spike=_one_key(where, where))
    w = a.want(0)
    picks = [(0, p) for p in sorted({where, where + 1, 599, 598, 512, 544}) if where <= p < 600]
    for splits in (None, 1, 5, 10):
        assert _rel(a.rows(picks, splits), w[[p for _, p in picks]]) < DT[dtype]
    if dtype == torch.bfloat16:
        lo = max(0, min(where, 600 - 90))
        got = a.tiles([(0, lo, 600), (1, 0, 40)])[0]
        assert _rel(got, w[lo:]) < DT[dtype]


@BOTH
def test_a_future_key_is_never_seen(dtype):
    """The key right after a row, with an enormous score, must not show."""
    def spike(i, q, k):
        k[100:] = 40.0 * torch.sign(k[100:])
    a = Attn((4, 4, 32, 32), dtype, [180], seed=7, spike=spike)
    w = a.want(0)
    assert _rel(a.rows([(0, 99), (0, 98)]), w[[99, 98]]) < DT[dtype]
    if dtype == torch.bfloat16:
        assert _rel(a.tiles([(0, 40, 120)])[0][:60], w[40:100]) < DT[dtype]


@BOTH
def test_scores_that_grow_along_the_keys(dtype):
    """Running maxima that rise with every tile, so that earlier partial results are rescaled again and again."""
    def spike(i, q, k):
        n = k.shape[0]
        k *= torch.linspace(0.1, 3.0, n)[:, None, None, None]
    a = Attn((2, 1, 64, 80), dtype, [500], seed=8, spike=spike, scale=0.6)
    w = a.want(0)
    assert _rel(a.rows([(0, 499), (0, 256)], 3), w[[499, 256]]) < DT[dtype]
    if dtype == torch.bfloat16:
        assert _rel(a.tiles([(0, 200, 500)])[0], w[200:]) < DT[dtype]


@BOTH
@pytest.mark.parametrize("diff,lam", [(0.0, 0.0), (0.8, 0.35), (0.3, -0.6), (0.1, 1.4)])
def test_map_weights(diff, lam, dtype):
    a = Attn((4, 2, 32, 48), dtype, [90], seed=9, diff=diff, lam=lam)
    w = a.want(0)
    assert _rel(a.rows([(0, 89), (0, 40)]), w[[89, 40]]) < DT[dtype]
    if dtype == torch.bfloat16:
        assert _rel(a.tiles([(0, 0, 90)])[0], w) < DT[dtype]


@BOTH
@pytest.mark.parametrize("shape", [(4, 2, 40, 56), (3, 3, 64, 128), (2, 1, 300, 24), (6, 1, 16, 16)])
def test_prologue(shape, dtype):
    """Norm per vector, temperature, cache rows; and the form without keys of its own."""
    _, da = _mods()
    H, G, dim, vdim = shape
    d, v = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    gen = _gen(3)
    n, eps, coef, every = 9, 1e-3, 0.4, 7
    pos = torch.tensor([0, 5, 6, 7, 13, 14, 90, 1000, 3], dtype=torch.int32)
    slots = torch.tensor([5, 70, 1, -1, 2, 3, 64, 127, 10], dtype=torch.int32)
    qw, kw = 1 + 0.2 * torch.randn(dim, generator=gen), 1 + 0.2 * torch.randn(dim, generator=gen)
    P = lambda w: torch.nn.functional.pad(w, (0, d - dim)).cuda()
    m = da.DiffAttention(H, G, dim, d, vdim, v, 1.0, 0.5, 0.2, eps, P(qw), P(kw), coef, float(every))
    q, k = torch.randn(n, H, 2, dim, generator=gen).to(dtype), torch.randn(n, G, 2, dim, generator=gen).to(dtype)
    val = torch.randn(n, G, vdim, generator=gen).to(dtype)
    padv = lambda t, w: torch.nn.functional.pad(t, (0, w - t.shape[-1])).reshape(n, -1)
    proj = torch.cat([padv(q, d), padv(k, d), padv(val, v), torch.randn(n, 16, generator=gen).to(dtype)], 1).cuda()
    kc, vc = torch.full((2, 64, m.k_width), 3.0, dtype=dtype).cuda(), torch.full((2, 64, m.v_width), 3.0, dtype=dtype).cuda()
    got = da.head_prep(proj, m, pos.cuda(), slots.cuda(), kc, vc).cpu()
    temp = ref.query_temperature(pos, coef, every)
    want_q = ref.rms(q.double(), eps) * qw.double() * temp[:, None, None, None]
    want_k = ref.rms(k.double(), eps) * kw.double()
    tol = 4e-3 if dtype == torch.bfloat16 else 1e-6
    assert _rel(got[..., :dim], want_q) < tol and not got[..., dim:].any()
    kc, vc = kc.cpu().view(128, G, 2, d), vc.cpu().view(128, G, v)
    for r, s in enumerate(slots.tolist()):
        if s >= 0:
            assert _rel(kc[s, ..., :dim], want_k[r]) < tol and torch.equal(vc[s, :, :vdim], val[r])
    untouched = [s for s in range(128) if s not in slots.tolist()]
    assert (kc[untouched] == 3).all() and (vc[untouched] == 3).all()
    m.k_w = None
    only_q = da.head_prep(torch.cat([proj[:, :m.q_width], proj[:, -16:]], 1), m, pos.cuda(), slots.cuda(), None, None).cpu()
    assert torch.equal(only_q, got)
    m.temp_every = 0.0
    assert _rel(da.head_prep(proj[:, :m.q_width], m, pos.cuda(), slots.cuda(), None, None).cpu()[..., :dim],
                ref.rms(q.double(), eps) * qw.double()) < tol
