"""Kernels of the head-mixed decoder family, each against its plain fp32 / fp64 statement
(``models/reference_cpu/rutulix_ref.py``)."""
import pytest
import torch

from deepseek_v4_2080ti_b200.models.reference_cpu import rutulix_ref as ref

pytestmark = pytest.mark.gpu
DT = {torch.bfloat16: 1.2e-2, torch.float32: 2e-6}


def _mods():
    from deepseek_v4_2080ti_b200.ops import _lib, mixattn
    return _lib, mixattn


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / b.norm().clamp_min(1e-30))


def _rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("cols,n", [(16, 3), (100, 5), (333, 2), (4096, 4), (8200, 2)])
def test_residual_norm(dtype, cols, n):
    _, mx = _mods()
    ld, eps = mx.pad16(cols), 1e-3
    pad = lambda t, dt: torch.nn.functional.pad(t, (0, ld - cols)).to("cuda", dt).contiguous()
    x, d = _rand(n, cols, seed=1) + 3.0, _rand(n, cols, seed=2).to(dtype).float()
    bias, post, step, pre = _rand(cols, seed=3), 1 + _rand(cols, seed=4, scale=0.2), _rand(cols, seed=5), 1 + _rand(cols, seed=6, scale=0.2)
    P = lambda v: pad(v, torch.float32)
    want_x = x.double() + ref.layer_norm(d.double() + bias.double(), post.double(), eps) + step.double()
    want_y = ref.layer_norm(want_x, pre.double(), eps)
    xg = pad(x, torch.float32)
    y = mx.residual_norm(xg, cols, eps, delta=pad(d, dtype), bias=P(bias), post_w=P(post), step=P(step), pre_w=P(pre))
    assert y.dtype == dtype and _rel(y[:, :cols], want_y) < DT[dtype] and _rel(xg[:, :cols], want_x) < 2e-6
    assert ld == cols or (not y[:, cols:].any() and not xg[:, cols:].any())
    # selected rows: the stored residual stays as it is
    keep = xg.clone()
    rows = torch.tensor([n - 1, 0], dtype=torch.int32, device="cuda")
    y2 = mx.residual_norm(xg, cols, eps, delta=pad(d, dtype), post_w=P(post), pre_w=P(pre), rows=rows)
    want = ref.layer_norm((want_x + ref.layer_norm(d.double(), post.double(), eps))[[n - 1, 0]], pre.double(), eps)
    assert _rel(y2[:, :cols], want) < DT[dtype] and torch.equal(keep, xg)
    # no norm on the way in; RMS norm with one-plus weights on the way out
    y3 = mx.residual_norm(xg, cols, eps, delta=pad(d, dtype), pre_w=P(pre - 1), rms=True, unit_offset=True)
    want = want_x + d.double()
    assert _rel(y3[:, :cols], ref.rms_norm(want, pre.double(), eps)) < DT[dtype] and _rel(xg[:, :cols], want) < 2e-6
    # nothing but the residual update
    assert mx.residual_norm(xg, cols, eps, delta=pad(d, dtype), post_w=P(post)) is None
    # start from an embedding table
    table, ids = _rand(7, cols, seed=8).to(dtype), torch.tensor([6, 0, 3, 3, 1][:n], dtype=torch.int32)
    y4 = mx.residual_norm(xg, cols, eps, ids=ids.cuda(), table=pad(table, dtype), step=P(step), pre_w=P(pre))
    want = table[ids.long()].double() + step.double()
    assert _rel(xg[:, :cols], want) < 2e-6 and _rel(y4[:, :cols], ref.layer_norm(want, pre.double(), eps)) < DT[dtype]


def test_layer_norm_of_a_row_with_a_large_mean():
    _, mx = _mods()
    x = (_rand(2, 512, seed=9) * 1e-2 + 50.0)
    one = torch.ones(512, device="cuda")
    y = mx.residual_norm(x.cuda(), 512, 1e-6, pre_w=one, dtype=torch.float32)
    assert _rel(y, ref.layer_norm(x.double(), torch.ones(512).double(), 1e-6)) < 1e-4


@pytest.mark.parametrize("dtype", list(DT))
def test_bias_xielu(dtype):
    _, mx = _mods()
    z = torch.cat([_rand(6, 40, seed=1, scale=3.0), torch.linspace(-90, 9, 40)[None], torch.linspace(-1e-3, 1e-3, 40)[None]])
    z = torch.nn.functional.pad(z, (0, 8)).to(dtype)
    bias = torch.nn.functional.pad(_rand(40, seed=2), (0, 8))
    act = torch.tensor([0.4, -1.1]).double()
    sp = torch.nn.functional.softplus(act)
    want = ref.xielu(z.double() + bias.double(), act)
    got = mx.bias_xielu(z.cuda(), bias.cuda(), float(sp[0]), float(0.5 + sp[1]))
    assert got.dtype == dtype and _rel(got, want) < DT[dtype] and not got[:, 40:].any()
    tiny = mx.bias_xielu(z[-1:].cuda(), None, float(sp[0]), float(0.5 + sp[1]))
    assert (tiny.double().cpu() - ref.xielu(z[-1:].double(), act)).abs().max() < (1e-9 if dtype == torch.float32 else 4e-6)


@pytest.mark.parametrize("t,n,k", [(1, 5, 16), (70, 100, 33), (65, 64, 128), (130, 257, 48)])
def test_gemm_f32(t, n, k):
    _, mx = _mods()
    x, w = _rand(t, k, seed=1), _rand(n, k, seed=2)
    assert _rel(mx.gemm_f32(x.cuda(), w.cuda()), x.double() @ w.double().t()) < 1e-6


def _mix(mx, H, G, dim, scale, chunk, rot, scaling=None, base=900.0, eps=1e-4, seed=0, dev="cuda"):
    """(HeadMix, unpadded q norm, k norm, talk)"""
    d = mx.pad8(dim)
    qn, kn = 1 + _rand(H * dim, seed=seed + 1, scale=0.3), 1 + _rand(G * dim, seed=seed + 2, scale=0.3)
    talk = torch.eye(H) + _rand(H, H, seed=seed + 3, scale=0.5)
    ph = lambda w, n: torch.nn.functional.pad(w.view(n, dim), (0, d - dim)).reshape(-1).contiguous().to(dev)
    tt = torch.zeros(H, (H + 3) // 4 * 4)
    tt[:, :H] = talk.t()
    freq, ms = mx.yarn_freqs(rot, base, scaling, dev)
    return mx.HeadMix(H, G, dim, d, scale, chunk, rot, freq, ms, eps, ph(qn, H), ph(kn, G), tt.to(dev)), qn, kn, talk


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
SIZES = [(6, 3, 32, 16), (4, 1, 24, 24), (5, 5, 20, 8), (3, 1, 10, 10), (8, 2, 128, 64), (4, 4, 200, 40), (16, 8, 64, 2), (2, 2, 256, 128),
         (1, 1, 16, 4)]


def _paged(rows, pages, bs, kw, dtype):
    """Zeroed cache + a scattered page list for `rows` positions."""
    perm = torch.randperm(pages - 1, generator=torch.Generator().manual_seed(rows))[: (rows + bs - 1) // bs] + 1
    return torch.zeros(pages, bs, kw, dtype=dtype, device="cuda"), torch.zeros(pages, bs, kw, dtype=dtype, device="cuda"), perm


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H,G,dim,rot", SIZES)
def test_qk_row_prep(dtype, H, G, dim, rot):
    _, mx = _mods()
    m, qn, kn, talk = _mix(mx, H, G, dim, 0.3, 0, rot, YARN if rot > 2 else None)
    t, n_mix, bs = 7, 0 if dtype == torch.float32 else 4, 16
    d, kw = m.d, G * m.d
    ph = lambda x, n: torch.nn.functional.pad(x.view(t, n, dim), (0, d - dim)).reshape(t, n * d)
    q, k = _rand(t, H * dim, seed=11).to(dtype), _rand(t, G * dim, seed=12).to(dtype)
    ld = mx.pad16((H + G) * d)
    proj = torch.zeros(t, ld, dtype=dtype, device="cuda")
    proj[:, :H * d], proj[:, H * d:H * d + kw] = ph(q, H), ph(k, G)
    pos = torch.tensor([0, 1, 5, 100, 4097, 70000, 12], dtype=torch.int32)
    kc, vc, _ = _paged(t, 5, bs, kw, dtype)
    slots = torch.tensor([17, 16, 40, 79, 33, 18, 64], dtype=torch.int32)
    q_mix, q_row = mx.qk_row_prep(proj, m, pos.cuda(), slots.cuda(), kc, vc, n_mix)
    freqs, ms = ref.yarn_frequencies(rot, 900.0, YARN if rot > 2 else None)
    full = lambda x, w, n: ref.rotate_interleaved(ref.rms_norm(x.double(), w.double(), m.eps).view(t, n, dim), pos, freqs, ms)
    wq, wk = full(q, qn, H), full(k, kn, G)
    got_k = kc.view(-1, kw)[slots.long().cuda()].view(t, G, d)
    got_v = vc.view(-1, kw)[slots.long().cuda()].view(t, G, d)
    assert _rel(got_k[..., :dim], wk) < DT[dtype] and torch.equal(got_v[..., :dim].cpu(), k.view(t, G, dim))
    assert not got_k[..., dim:].any() and int((kc != 0).any(-1).sum()) == t
    assert _rel(q_row[..., :dim], wq[n_mix:]) < 2e-6 and not q_row[..., dim:].any()
    if n_mix:
        want = torch.einsum("hcr,tcrd->thcd", talk.double().view(H, G, H // G), wq[:n_mix].view(n_mix, G, H // G, dim))
        got = q_mix.view(n_mix, H, G, d)
        assert _rel(got[..., :dim], want) < 5e-3 and not got[..., dim:].any()


def _setup_attention(mx, H, G, dim, chunk, lens, dtype, bs=16, seed=0, scale=0.4):
    """Sequences of the given lengths in one scattered cache; returns everything both kernels need."""
    m, *_, talk = _mix(mx, H, G, dim, scale, chunk, 0, seed=seed)
    d, kw = m.d, G * m.d
    pages = 1 + sum((n + bs - 1) // bs for n in lens)
    order = (torch.randperm(pages - 1, generator=torch.Generator().manual_seed(seed)) + 1).tolist()
    width = max((n + bs - 1) // bs for n in lens) + 2
    table = torch.zeros(len(lens), width, dtype=torch.int32)
    # pages hold finite junk past the sequences' ends and in page 0, as after reuse
    kc, vc = (torch.randn(pages, bs, kw, generator=torch.Generator().manual_seed(seed + i)).mul(30).to("cuda", dtype) for i in (50, 51))
    seqs = []
    for s, n in enumerate(lens):
        q = _rand(n, H, dim, seed=100 + 7 * s + seed)
        k, v = _rand(n, G, dim, seed=101 + 7 * s + seed).to(dtype).float(), _rand(n, G, dim, seed=102 + 7 * s + seed).to(dtype).float()
        seqs.append([q, k, v])
        for b in range((n + bs - 1) // bs):
            table[s, b] = order.pop()

    def load():
        for s, (q, k, v) in enumerate(seqs):
            for c, x in ((kc, k), (vc, v)):
                xp = torch.nn.functional.pad(x, (0, d - dim)).reshape(len(x), kw).to("cuda", dtype)
                for b in range((len(x) + bs - 1) // bs):
                    part = xp[b * bs:(b + 1) * bs]
                    c[int(table[s, b]), :len(part)] = part
    return m, talk, kc, vc, table, seqs, load


def _want(m, talk, q, k, v, scale, chunk):
    f = lambda x: x.double()
    return ref.talking_attention(f(q), f(k), f(v), f(talk), scale, ref.chunk_visible(len(q), chunk or None)).reshape(len(q), -1)


def _run_rows(mx, m, talk, kc, vc, table, seqs, picks, dtype, splits):
    """picks: (sequence, position) per row."""
    pad = lambda x: torch.nn.functional.pad(x, (0, m.d - m.dim))
    q = torch.stack([pad(seqs[s][0][p]) for s, p in picks]).cuda().contiguous()
    out = torch.zeros(len(picks), mx.pad16(m.heads * m.d), dtype=dtype, device="cuda")
    mx.rows(q, m, kc, vc, table.cuda(), torch.tensor([p for _, p in picks], dtype=torch.int32, device="cuda"), 1 << 12, out,
            seq=torch.tensor([s for s, _ in picks], dtype=torch.int32, device="cuda"), splits=splits)
    return out[:, :m.heads * m.d].view(len(picks), m.heads, m.d)[..., :m.dim].reshape(len(picks), -1)


def _run_tiles(mx, m, talk, kc, vc, table, seqs, portions):
    """portions: (sequence, first position, tokens) per entry; keys up to the portion's end are in the cache."""
    rows, starts = [], []
    for s, p0, n in portions:
        starts.append(sum(r.shape[0] for r in rows))
        rows.append(seqs[s][0][p0:p0 + n])
    q = torch.cat(rows).cuda()
    H, G, R = m.heads, m.groups, m.heads // m.groups
    mixed = torch.einsum("hcr,tcrd->thcd", talk.cuda().view(H, G, R), q.view(-1, G, R, m.dim))
    q_mix = torch.nn.functional.pad(mixed, (0, m.d - m.dim)).reshape(-1, H, G * m.d).bfloat16().contiguous()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    out = torch.zeros(q.shape[0], mx.pad16(H * m.d), dtype=torch.bfloat16, device="cuda")
    mx.prefill(q_mix, m, kc, vc, table.cuda(), i32(starts), i32([n for *_, n in portions]), i32([p + n for _, p, n in portions]),
               max(n for *_, n in portions), out, seq=i32([s for s, *_ in portions]))
    return out[:, :H * m.d].view(-1, H, m.d)[..., :m.dim].reshape(q.shape[0], -1)


@pytest.mark.parametrize("dtype", list(DT))
@pytest.mark.parametrize("H,G,dim,_rot", SIZES)
@pytest.mark.parametrize("chunk", [0, 37])
def test_row_attention(dtype, H, G, dim, _rot, chunk):
    lib, mx = _mods()
    lens = [1, 40, 150]
    m, talk, kc, vc, table, seqs, load = _setup_attention(mx, H, G, dim, chunk, lens, dtype)
    load()
    picks = [(0, 0), (1, 39), (1, 36), (1, 37), (2, 149), (2, 73), (2, 74), (2, 0), (2, 111), (2, 110), (2, 16), (2, 15)]
    want = torch.stack([_want(m, talk, *seqs[s], m.scale, chunk)[p] for s, p in picks])
    for splits in (1, 2, 5):
        got = _run_rows(mx, m, talk, kc, vc, table, seqs, picks, dtype, splits)
        lib.check_status()
        assert _rel(got, want) < (5e-3 if dtype == torch.bfloat16 else 1e-5), splits
        assert max(_rel(g, w) for g, w in zip(got, want)) < (1e-2 if dtype == torch.bfloat16 else 2e-5)


@pytest.mark.parametrize("H,G,dim,_rot", SIZES + [(8, 8, 128, 0), (32, 8, 128, 0)])
@pytest.mark.parametrize("chunk,bs", [(0, 64), (37, 16), (130, 64), (128, 128)])
def test_tile_attention(H, G, dim, _rot, chunk, bs):
    lib, mx = _mods()
    if not mx._lib.lib().b200_attn_mix_prefill_supported(H, G, mx.pad8(dim), bs):
        pytest.skip("covered by the row kernel")
    lens = [300, 20, 131]
    m, talk, kc, vc, table, seqs, load = _setup_attention(mx, H, G, dim, chunk, lens, torch.bfloat16, bs=bs, scale=0.15)
    load()
    for portions in ([(0, 0, 300)], [(0, 290, 10), (1, 0, 20), (2, 1, 130)], [(2, 129, 2), (0, 36, 150)]):
        # the cache also holds later positions than the portion's end; they must stay invisible
        got = _run_tiles(mx, m, talk, kc, vc, table, seqs, portions)
        lib.check_status()
        want = torch.cat([_want(m, talk, *seqs[s], m.scale, chunk)[p:p + n] for s, p, n in portions])
        assert _rel(got, want) < 1e-2, portions
        worst = max(_rel(g, w) for g, w in zip(got, want))
        assert worst < 4e-2, (portions, worst)


@pytest.mark.parametrize("kernel", ["rows", "tiles"])
@pytest.mark.parametrize("chunk,size", [(48, 200), (64, 200), (100, 260), (0, 200)])
def test_one_score_that_stands_out_is_seen_exactly_inside_the_chunk(kernel, chunk, size):
    """A key aligned with the query dominates the softmax when it is visible and leaves no trace when it is not: the first
    position of the chunk, the last of the one before, page borders, far keys."""
    lib, mx = _mods()
    H, G, dim, bs = 4, 2, 32, 16
    m, talk, kc, vc, table, seqs, load = _setup_attention(mx, H, G, dim, chunk, [size], torch.bfloat16, bs=bs, seed=4)
    talk = torch.eye(H)
    m.talk_t.copy_(torch.eye(H))
    q, k, v = seqs[0]
    q.mul_(0.3)
    k.mul_(0.3)
    base_k = k.clone()
    i = size - 7
    lo = i - i % chunk if chunk else 0
    mark = torch.full((dim,), 3.0)
    q[i] = mark
    for j in sorted({lo, lo - 1, lo + 1, i, i - 1, 0, bs * 9, bs * 9 - 1, 128, 127} & set(range(i + 1))):
        k.copy_(base_k)
        k[j, :] = mark
        load()
        got = (_run_rows(mx, m, talk, kc, vc, table, seqs, [(0, i)], torch.bfloat16, 2)[0] if kernel == "rows"
               else _run_tiles(mx, m, talk, kc, vc, table, seqs, [(0, i - 20, 27)])[20])
        want = _want(m, talk, q, k, v, m.scale, chunk)[i]
        assert _rel(got, want) < 1e-2, j
        seen = _rel(got, v[j].repeat_interleave(H // G, 0).reshape(-1)) < 2e-2
        assert seen == (lo <= j <= i), j
    lib.check_status()


def test_rows_do_not_depend_on_batch_splits_or_pages():
    _, mx = _mods()
    m, talk, kc, vc, table, seqs, load = _setup_attention(mx, 6, 3, 32, 0, [90, 120], torch.float32)
    load()
    both = _run_rows(mx, m, talk, kc, vc, table, seqs, [(0, 80), (1, 119), (0, 3)], torch.float32, 3)
    for r, pick in enumerate([(0, 80), (1, 119), (0, 3)]):
        for splits in (1, 3, 64):
            alone = _run_rows(mx, m, talk, kc, vc, table, seqs, [pick], torch.float32, splits)
            assert _rel(alone[0], both[r]) < 2e-6


def test_workspace_growth_keeps_captured_addresses_alive():
    _, mx = _mods()
    before = mx._ws.get(0)
    m, talk, kc, vc, table, seqs, load = _setup_attention(mx, 4, 4, 200, 0, [64], torch.bfloat16)
    load()
    _run_rows(mx, m, talk, kc, vc, table, seqs, [(0, p) for p in range(60)], torch.bfloat16, 64)
    now = mx._ws[0]
    assert before is None or now is before or any(t is before for t in mx._outgrown)


@pytest.mark.parametrize("t,n,k", [(3, 320, 192), (5, 96, 4096), (40, 256, 2048), (128, 128, 512), (300, 144, 80), (256, 512, 128), (512, 256, 1024)])
def test_projection_with_activation_in_the_epilogue(t, n, k):
    """Every route of the bf16 GEMM: one pass, split K with the reducing CTA, token tiles of all sizes, CTA pairs."""
    lib, _ = _mods()
    from deepseek_v4_2080ti_b200.ops import gemm
    x, w = _rand(t, k, seed=1).bfloat16(), (_rand(n, k, seed=2) * 2 / k ** 0.5).bfloat16()
    bias, act = _rand(n, seed=3), torch.tensor([0.2, -0.4]).double()
    sp = torch.nn.functional.softplus(act)
    got = gemm.linear_bias_xielu(x.cuda(), gemm.PackedLinear.from_bf16(w.cuda()), bias.cuda(), float(sp[0]), float(0.5 + sp[1]))
    lib.check_status()
    z = x.double() @ w.double().t() + bias.double()
    assert _rel(got, ref.xielu(z, act)) < 4e-3
    # a following plain product is not affected by the activation of this one
    assert _rel(gemm.linear(x.cuda(), gemm.PackedLinear.from_bf16(w.cuda())), x.double() @ w.double().t()) < 4e-3
