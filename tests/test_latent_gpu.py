"""Latent-attention kernels against the plain statement: prologue and cache append, rotation, per-head products, gathered
contexts, single rows in the absorbed form and prompt tiles over expanded keys, with single scores that stand out at page and
tile borders, far keys, and the first tokens."""
import pytest
import torch

from deepseek_v4_2080ti_b200.models.reference_cpu import kemirax_ref as ref

pytestmark = pytest.mark.gpu
DT = {torch.bfloat16: 1e-2, torch.float32: 3e-6}
BOTH = pytest.mark.parametrize("dtype", list(DT))
YARN = {"factor": 5.0, "original": 128, "fast": 6.0, "slow": 1.0}


def _mods():
    from deepseek_v4_2080ti_b200.ops import _lib, latent
    return _lib, latent


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-30))


def _pad(n):
    return (n + 15) // 16 * 16


def _i32(v):
    return torch.tensor(v, dtype=torch.int32).cuda()


def _mixer(heads, dim, rot, vdim, q_rank, kv_rank, scale=0.2, rot_dims=None, base=3000.0, yarn=YARN, own=True, seed=0, eps=1e-4):
    _, lat = _mods()
    gen = torch.Generator().manual_seed(seed)
    rd = rot if rot_dims is None else rot_dims
    spec = {"dims": rd, "base": base, "scaling": yarn}
    freq, ms = ref.yarn_frequencies(spec)
    qw, cw = torch.zeros(_pad(q_rank)), torch.zeros(_pad(kv_rank))
    qw[:q_rank], cw[:kv_rank] = 1 + 0.3 * torch.randn(q_rank, generator=gen), 1 + 0.3 * torch.randn(kv_rank, generator=gen)
    m = lat.LatentAttention(heads, dim, _pad(dim), rot, _pad(rot), vdim, _pad(vdim), q_rank, _pad(q_rank), kv_rank, _pad(kv_rank), scale, eps,
                            rd, freq.cuda(), ms, qw.cuda(), cw.cuda() if own else None)
    return m, spec


SIZES = [  # heads, dim, rot, vdim, q_rank, kv_rank
    (5, 12, 6, 18, 20, 28), (2, 64, 16, 64, 48, 64), (16, 128, 64, 128, 96, 512), (20, 32, 8, 48, 33, 144), (40, 16, 2, 16, 16, 96)]


@BOTH
@pytest.mark.parametrize("own", [True, False])
@pytest.mark.parametrize("sizes", SIZES[:4])
def test_prologue(dtype, own, sizes):
    _, lat = _mods()
    heads, dim, rot, vdim, qr, kr = sizes
    rd = rot if own else rot - 2                    # part of the key may pass unrotated
    m, spec = _mixer(*sizes, rot_dims=rd if rd > 0 else rot, own=own, seed=1)
    n, gen = 9, torch.Generator().manual_seed(2)
    zq, zc, zr = (torch.randn(n, k, generator=gen).to(dtype) for k in (qr, kr, rot))
    proj = torch.zeros(n, m.q_pad + (m.c + m.r if own else 0) + 32, dtype=dtype)
    proj[:, :qr] = zq
    if own:
        proj[:, m.q_pad:m.q_pad + kr], proj[:, m.q_pad + m.c:m.q_pad + m.c + rot] = zc, zr
    proj[:, -32:] = 99.0
    pos = [0, 1, 63, 64, 500, 7, 100000, 3, 2]
    slots = [70, 3, 4, 64, 127, 128, 191, 66, 90]
    cache = torch.full((4, 64, m.cache_width), 7.0, dtype=dtype).cuda()
    got = lat.prep(proj.cuda(), m, _i32(pos), _i32(slots), cache)
    want = ref.rms(zq.double(), m.eps) * m.q_w[:qr].double().cpu()
    assert _rel(got[:, :qr], want) < DT[dtype] and not got[:, qr:].any()
    if not own:
        assert bool((cache == 7).all())
        return
    rows = cache.view(-1, m.cache_width)[slots].cpu()
    assert _rel(rows[:, :kr], ref.rms(zc.double(), m.eps) * m.c_w[:kr].double().cpu()) < DT[dtype] and not rows[:, kr:m.c].any()
    # a far position turns the fast pairs thousands of times: the angle itself must be exact
    assert _rel(rows[:, m.c:m.c + rot], ref.rotate_half(zr.double(), pos, spec)) < DT[dtype] and not rows[:, m.c + rot:].any()
    others = [i for i in range(256) if i not in slots]
    assert bool((cache.view(-1, m.cache_width)[others] == 7).all())


@BOTH
def test_rotation_in_place_and_into_another_layout(dtype):
    _, lat = _mods()
    m, spec = _mixer(3, 12, 10, 16, 16, 32, rot_dims=6, seed=3)
    n, w, gen = 7, 16 + 16, torch.Generator().manual_seed(4)
    q = torch.zeros(n, 3 * w + 16, dtype=dtype)
    v = torch.randn(n, 3, 10, generator=gen).to(dtype)
    nope = torch.randn(n, 3, 16, generator=gen).to(dtype)
    q[:, :3 * w].view(n, 3, w)[:, :, :16], q[:, :3 * w].view(n, 3, w)[:, :, 16:26] = nope, v
    pos = list(range(40, 47))
    want = ref.rotate_half(v.double(), pos, spec)
    out = torch.full((n, 3, 60), 5.0, dtype=dtype).cuda()
    g = q.cuda()
    lat.rotate_heads(g, m, _i32(pos), out, 44)
    assert torch.equal(g.cpu(), q) and bool((out[:, :, :44] == 5).all()) and _rel(out[:, :, 44:54], want) < DT[dtype] and not out[:, :, 54:].any()
    lat.rotate_heads(g, m, _i32(pos))
    h = g[:, :3 * w].view(n, 3, w).cpu()
    assert torch.equal(h[:, :, :16], nope) and _rel(h[:, :, 16:26], want) < DT[dtype] and not g[:, 3 * w:].any()


@BOTH
@pytest.mark.parametrize("t,h,n,k", [(1, 3, 16, 16), (5, 2, 48, 80), (33, 4, 128, 512), (17, 16, 512, 128), (70, 1, 30, 176), (200, 2, 64, 32)])
def test_products_per_head(dtype, t, h, n, k):
    _, lat = _mods()
    gen = torch.Generator().manual_seed(t)
    x, w = torch.randn(t, h, k + 16, generator=gen).to(dtype), torch.randn(h, n, k, generator=gen).to(dtype)
    y = torch.full((t, h, n + 8 if n % 8 == 0 else n + 2), 3.0, dtype=dtype).cuda()
    ldy = y.shape[2]
    if dtype == torch.bfloat16 and (ldy % 8):
        y = torch.full((t, h, 40), 3.0, dtype=dtype).cuda()
        ldy = 40
    xc = x.cuda()
    lat.head_linear(xc[:, :, 16:], xc.stride(0), k + 16, w.cuda(), y, h * ldy, ldy, t)
    assert _rel(y[:, :, :n], torch.einsum("thk,hnk->thn", x[:, :, 16:].double(), w.double())) < DT[dtype]
    assert bool((y[:, :, n:] == 3).all())


class Ctx:
    """Random cache rows of several sequences over shuffled pages, unread memory poisoned."""

    def __init__(self, m, lengths, dtype, block=64, seed=0):
        gen = torch.Generator().manual_seed(seed)
        self.m, self.dtype, self.block = m, dtype, block
        self.c = [torch.randn(n, m.kv_rank, generator=gen).to(dtype) for n in lengths]
        self.kr = [torch.randn(n, m.rot_dim, generator=gen).to(dtype) for n in lengths]
        pages = [(n + block - 1) // block for n in lengths]
        order = torch.randperm(sum(pages), generator=gen) + 1
        self.table = torch.zeros(len(lengths), max(pages) + 2, dtype=torch.int32)
        self.cache = torch.full((sum(pages) + 1, block, m.cache_width), 3.0, dtype=dtype)
        at = 0
        for i, n in enumerate(lengths):
            self.table[i, :pages[i]] = order[at:at + pages[i]].to(torch.int32)
            at += pages[i]
            for p in range(n):
                row = self.cache[self.table[i, p // block], p % block]
                row.zero_()
                row[:m.kv_rank], row[m.c:m.c + m.rot_dim] = self.c[i][p], self.kr[i][p]
        self.table[:, -2:] = 0
        self.gcache, self.gtable = self.cache.cuda(), self.table.cuda()

    def loud(self, i, p, q):
        """Key p of sequence i lines up with absorbed query q [c | r] and beats the others by a wide margin."""
        c, r = self.m.kv_rank, self.m.rot_dim
        s = 30.0 / float(self.m.scale * (q[:c].double().pow(2).sum() + q[self.m.c:self.m.c + r].double().pow(2).sum()))
        self.c[i][p], self.kr[i][p] = (q[:c] * s).to(self.dtype), (q[self.m.c:self.m.c + r] * s).to(self.dtype)
        row = self.cache[self.table[i, p // self.block], p % self.block]
        row[:c], row[self.m.c:self.m.c + r] = self.c[i][p], self.kr[i][p]
        self.gcache = self.cache.cuda()


def _absorbed(m, n, dtype, seed):
    q = torch.zeros(n, m.heads, m.cache_width)
    gen = torch.Generator().manual_seed(seed)
    q[:, :, :m.kv_rank] = torch.randn(n, m.heads, m.kv_rank, generator=gen) * m.kv_rank ** -0.5
    q[:, :, m.c:m.c + m.rot_dim] = torch.randn(n, m.heads, m.rot_dim, generator=gen) * m.rot_dim ** -0.5
    return q.to(dtype)


def _attend(m, q, c, kr, pos):
    """One row: q [heads, c + r] over keys up to ``pos``."""
    s = (q[:, :m.kv_rank].double() @ c[:pos + 1].double().t() + q[:, m.c:m.c + m.rot_dim].double() @ kr[:pos + 1].double().t()) * m.scale
    return torch.softmax(s, -1) @ c[:pos + 1].double()


@pytest.mark.parametrize("dtype,tiles", [(torch.bfloat16, True), (torch.bfloat16, False), (torch.float32, False)])
@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("splits", [None, 1, 7])
def test_single_rows(dtype, tiles, sizes, splits):
    """Rows of several sequences at positions around page and tile borders, first tokens included; one key per head stands out,
    wherever it lies, also when it is the row's own or the very first."""
    _lib, lat = _mods()
    m, _ = _mixer(*sizes, scale=1.3, seed=5)
    ctx = Ctx(m, [300, 65, 1, 130], dtype, block=32, seed=6)
    where = [(0, 299), (0, 0), (0, 31), (0, 32), (1, 64), (2, 0), (3, 127), (3, 128), (0, 200)]
    q = _absorbed(m, len(where), dtype, 7)
    got = lat.attend_rows(q.cuda(), m, ctx.gcache, ctx.gtable, _i32([p for _, p in where]), 301, seq=_i32([i for i, _ in where]), splits=splits,
                          tiles=tiles)
    _lib.check_status()
    if tiles:
        assert _lib.lib().b200_attn_latent_decode_heads(m.heads, m.c, m.cache_width, 32) > 0
    for r, (i, p) in enumerate(where):
        assert _rel(got[r, :, :m.kv_rank], _attend(m, q[r], ctx.c[i], ctx.kr[i], p)) < DT[dtype], (r, i, p)
    assert not got[:, :, m.kv_rank:].any()
    for far in (0, 31, 32, 63, 150, 299):
        ctx = Ctx(m, [300, 65, 1, 130], dtype, block=32, seed=6)
        ctx.loud(0, far, q[0, m.heads - 1])
        rows = [p for p in (far - 1, far, 299) if p >= 0]
        qq = q[:1].expand(len(rows), -1, -1).contiguous()
        got = lat.attend_rows(qq.cuda(), m, ctx.gcache, ctx.gtable[:1].expand(len(rows), -1).contiguous(), _i32(rows), 301, splits=splits, tiles=tiles)
        for r, p in enumerate(rows):
            want = _attend(m, qq[r], ctx.c[0], ctx.kr[0], p)
            assert _rel(got[r, :, :m.kv_rank], want) < 2 * DT[dtype], (far, p)
            seen = _rel(want[-1], ctx.c[0][far].double()) < 0.05
            assert seen == (p >= far)                        # the test itself tells a missed or a leaked key apart


@pytest.mark.parametrize("block", [16, 32, 64, 128])
@pytest.mark.parametrize("heads,kv_rank,rot", [(16, 512, 64), (5, 48, 32), (33, 208, 16), (50, 448, 64)])
def test_single_rows_over_long_contexts(block, heads, kv_rank, rot):
    """Growing scores (every tile moves the running maximum), all page sizes, one to four accumulators, several head groups."""
    _lib, lat = _mods()
    m, _ = _mixer(heads, 16, rot, 16, 16, kv_rank, scale=0.9, seed=15)
    ctx = Ctx(m, [1500, 200], torch.bfloat16, block=block, seed=16)
    q = _absorbed(m, 3, torch.bfloat16, 17)
    ramp = torch.linspace(0.05, 4.0, 1500)[:, None]
    for p in range(1500):
        ctx.c[0][p] = (ctx.c[0][p].float() * 0.3 + q[0, p % heads, :kv_rank].float() * ramp[p] * kv_rank ** 0.5).bfloat16()
        row = ctx.cache[ctx.table[0, p // block], p % block]
        row[:kv_rank] = ctx.c[0][p]
    ctx.gcache = ctx.cache.cuda()
    for splits in (None, 1, 3, 40):
        got = lat.attend_rows(q.cuda(), m, ctx.gcache, ctx.gtable, _i32([1499, 700, 199]), 1500, seq=_i32([0, 0, 1]), splits=splits)
        _lib.check_status()
        for r, (i, p) in enumerate(((0, 1499), (0, 700), (1, 199))):
            assert _rel(got[r, :, :kv_rank], _attend(m, q[r], ctx.c[i], ctx.kr[i], p)) < 1e-2, (splits, r)


@pytest.mark.parametrize("block", [16, 64])
def test_gathered_contexts(block):
    _, lat = _mods()
    m, _ = _mixer(2, 16, 6, 16, 16, 40, seed=8)
    ctx = Ctx(m, [70, 3, 129], torch.bfloat16, block=block, seed=9)
    starts = [0, 129, 132]
    c, k = lat.gather(ctx.gcache, m, ctx.gtable, _i32([2, 1, 0]), _i32([129, 3, 70]), _i32(starts), 202)
    assert c.shape == (256, 48) and k.shape == (256, 64)
    for s, i, n in zip(starts, (2, 1, 0), (129, 3, 70)):
        assert torch.equal(c[s:s + n, :40].cpu(), ctx.c[i][:n]) and torch.equal(k[s:s + n, :6].cpu(), ctx.kr[i][:n])
    assert not c[202:].any() and not k[202:].any() and not c[:, 40:].any() and not k[:, 6:].any()


TILE_SIZES = [  # heads, dim, rot, vdim, q_rank, kv_rank: one to four key slabs, one and two value slabs, sliced values
    (3, 20, 6, 28, 16, 64), (2, 128, 64, 128, 16, 128), (2, 64, 16, 64, 16, 64), (2, 80, 64, 96, 16, 48), (1, 192, 64, 128, 16, 64),
    (2, 48, 32, 200, 16, 32), (2, 64, 64, 32, 16, 512)]


@pytest.mark.parametrize("sizes", TILE_SIZES)
@pytest.mark.parametrize("limit", [1 << 29, 1 << 14])
def test_prompt_tiles(sizes, limit, monkeypatch):
    """Portions of several sequences at once, long and short contexts before them, queries that single one key out at tile,
    stream and portion borders; also in several rounds of heads."""
    _lib, lat = _mods()
    from deepseek_v4_2080ti_b200.ops import gemm
    monkeypatch.setattr(lat, "EXPANDED_LIMIT", limit)
    m, _ = _mixer(*sizes, scale=0.35, seed=10)
    assert lat.tiles_supported(m)
    bf = torch.bfloat16
    entries = [(700, 700), (300, 40), (257, 129), (1, 1), (900, 2)]          # context length, own rows
    ctx = Ctx(m, [n for n, _ in entries], bf, seed=11)
    gen = torch.Generator().manual_seed(12)
    uk = torch.zeros(m.heads, m.d, m.c)
    uv = torch.zeros(m.heads, m.v, m.c)
    uk[:, :m.dim, :m.kv_rank] = torch.randn(m.heads, m.dim, m.kv_rank, generator=gen) * m.kv_rank ** -0.5
    uv[:, :m.vdim, :m.kv_rank] = torch.randn(m.heads, m.vdim, m.kv_rank, generator=gen) * m.kv_rank ** -0.5
    uk, uv = uk.to(bf), uv.to(bf)
    w = gemm.PackedLinear.from_bf16(torch.cat([uk, uv], 1).reshape(-1, m.c).cuda())
    rows = sum(n for _, n in entries)
    q = torch.zeros(rows, m.heads, m.head_width)
    q[:, :, :m.dim] = torch.randn(rows, m.heads, m.dim, generator=gen)
    q[:, :, m.d:m.d + m.rot_dim] = torch.randn(rows, m.heads, m.rot_dim, generator=gen)
    # rows whose query is one key's own direction, scaled up: (entry, row of the entry, key position)
    keys = [(c[:, :m.kv_rank].double() @ uk[:, :m.dim, :m.kv_rank].double().transpose(1, 2)).to(bf).double()
            for c in (ctx.c[i] for i in range(len(entries)))]                 # [heads, n, dim]
    first = [sum(n for _, n in entries[:i]) for i in range(len(entries))]
    aimed = [(0, 0, 0), (0, 127, 0), (0, 128, 127), (0, 129, 128), (0, 130, 130), (0, 255, 256), (0, 256, 255), (0, 511, 128), (0, 698, 0), (0, 699, 699),
             (0, 640, 641), (1, 0, 260), (1, 39, 128), (1, 5, 0), (2, 128, 256), (2, 0, 127), (4, 1, 0), (4, 0, 899)]
    for e, r, key in aimed:
        k = torch.cat([keys[e][:, key], ctx.kr[e][key].double().expand(m.heads, -1)], -1)
        k = k * (30.0 / m.scale / k.pow(2).sum(-1, keepdim=True))
        q[first[e] + r, :, :m.dim], q[first[e] + r, :, m.d:m.d + m.rot_dim] = k[:, :m.dim], k[:, m.dim:]
    q = q.to(bf)
    qd = torch.zeros(rows, m.heads * m.head_width + 16, dtype=bf)
    qd[:, :m.heads * m.head_width] = q.view(rows, -1)
    starts = [sum(n for n, _ in entries[:i]) for i in range(len(entries))]
    total = sum(n for n, _ in entries)
    kv_len, own, seq = _i32([n for n, _ in entries]), _i32([n for _, n in entries]), _i32(list(range(len(entries))))
    out = torch.full((rows, m.heads * m.v + 16), 5.0, dtype=bf).cuda()
    c, kr = lat.gather(ctx.gcache, m, ctx.gtable, seq, kv_len, _i32(starts), total)
    lat.attend_tiles(qd.cuda(), m, c, kr, w, _i32(first), own, kv_len, _i32(starts), max(n for _, n in entries), out)
    _lib.check_status()
    got = out[:, :m.heads * m.v].view(rows, m.heads, m.v).cpu().double()
    assert bool((out[:, m.heads * m.v:] == 5).all())
    for e, (n, mine) in enumerate(entries):
        vals = (ctx.c[e].double() @ uv[:, :m.vdim, :m.kv_rank].double().transpose(1, 2)).to(bf).double()
        qe = q[first[e]:first[e] + mine].double()
        s = torch.einsum("rhd,hnd->rhn", qe[:, :, :m.dim], keys[e]) + torch.einsum("rhd,nd->rhn", qe[:, :, m.d:m.d + m.rot_dim], ctx.kr[e].double())
        hidden = torch.arange(n)[None] > (n - mine + torch.arange(mine))[:, None]
        want = torch.einsum("rhn,hnv->rhv", torch.softmax((s * m.scale).masked_fill(hidden[:, None], float("-inf")), -1), vals)
        g = got[first[e]:first[e] + mine]
        assert _rel(g[:, :, :m.vdim], want) < 1e-2 and not g[:, :, m.vdim:].any()
        worst = (g[:, :, :m.vdim] - want).norm(dim=-1) / want.norm(dim=-1)
        assert float(worst.max()) < 4e-2, (e, int(worst.max(-1).values.argmax()))
        for r, key in ((r, k) for x, r, k in aimed if x == e and k <= n - mine + r):
            assert _rel(got[first[e] + r, 0, :m.vdim], vals[0, key]) < 5e-2, (e, r, key)      # the aimed key is what comes out


def test_sizes_outside_the_tile_kernel():
    _, lat = _mods()
    assert not lat.tiles_supported(_mixer(2, 200, 70, 64, 16, 64)[0])        # six slabs of keys
    assert lat.tiles_supported(_mixer(2, 130, 64, 64, 16, 64)[0])
