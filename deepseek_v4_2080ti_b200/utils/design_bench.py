"""Prefill and decode throughput of one decoder design at sizes of real models' layers (random weights), beside the
framework's closest existing model at equal size, and the kernels of both beside their rooflines.

    python bench.py --design rutulix|zigasun|kemirax|nunosun [--design-size small|large] [--steps K] [--warmup W]

Closest model of Rutulix: the Qwen-style decoder with full-attention layers only (per-head QK norm, grouped attention, SwiGLU
with FP8 weights) of the same width, heads and feed-forward parameters.  Of Zigasun: the same decoder with Gated-DeltaNet and
full-attention layers in turn (both recurrent states as wide as the scan's channels).  Of Kemirax: the latent-attention
decoder with routed experts, equal width, heads, latents and experts; its recurrence stands beside Gated DeltaNet.  Of Nunosun:
the Qwen-style decoder with Gated-DeltaNet and full-attention layers in turn, equal width, heads, recurrent channels and
feed-forward parameters per token.  Whole-model numbers: CUDA events around a prompt of
``--prompt`` tokens and around replayed decode steps.  Kernel numbers: CUDA events around single launches, L2 flushed
before each; fractions of the measured copy bandwidth / bf16 GEMM burst of MEASURED_PEAKS.json.
"""
from __future__ import annotations

import json
import os

import torch

PEAKS_FALLBACK = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
# Rutulix: width, heads, kv heads, head dim, SwiGLU width of the closest model (the two-matrix feed-forward gets 3/2 of it), chunk
SIZES = {"small": (2048, 16, 4, 128, 5632, 2048), "large": (4096, 32, 8, 128, 10752, 8192)}
# Zigasun: width, heads, kv heads, dim per map, value dim, feed-forward, scan channels, states, dt rank
ZG_SIZES = {"small": (2048, 16, 4, 64, 128, 5632, 4096, 16, 128), "large": (4096, 32, 8, 64, 128, 10752, 8192, 16, 256)}
# Kemirax: width, heads, dim, rotated dim, value dim, query latent, latent, linear-attention heads (128 x 128), expert and shared
# width, experts, identity experts, experts per token
KX_SIZES = {"small": (2048, 16, 128, 64, 128, 768, 512, 16, 1024, 64, 8, 6), "large": (4096, 32, 128, 64, 128, 1536, 512, 32, 1536, 128, 16, 8)}
KX_LAYERS = "gaba"
# Nunosun: width, heads, kv heads (128 x 128), window, retention heads (128 x 128), delta-rule heads and query / key heads
# (128 x 128), SwiGLU width of the closest model (the two-matrix feed-forward gets 3/2 of it, the experts of a token together
# as much), experts, experts per token, side embedding
NS_SIZES = {"small": (2048, 16, 4, 2048, 16, 32, 16, 5632, 64, 8, 256), "large": (4096, 32, 8, 4096, 32, 64, 16, 10752, 128, 8, 256)}
NS_LAYERS = "dpdp"
LAYERS, VOCAB = 4, 32768


def _peaks() -> tuple[dict, str]:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            return json.load(f), "of measured"
    except OSError:
        return PEAKS_FALLBACK, "of fallback"


class _Timer:
    def __init__(self, dev, steps: int, warmup: int):
        self.steps, self.warmup = max(3, steps), max(3, warmup)
        self.flush = torch.empty(96 << 20, dtype=torch.int32, device=dev)       # 384 MB, larger than L2

    def __call__(self, fn, flush: bool = True) -> float:
        """Median milliseconds of one call."""
        ms = []
        for i in range(self.warmup + self.steps):
            if flush:
                self.flush.fill_(i)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            if i >= self.warmup:
                ms.append(a.elapsed_time(b))
        return sorted(ms)[len(ms) // 2]


def _models(size: str, dev, prompt: int, slots: int):
    from ..models import qwen_hybrid as qh
    from ..models import rutulix as rx
    width, heads, kv, dim, inter, chunk = SIZES[size]
    cfg = rx.RutulixConfig.uniform(LAYERS, width, heads, kv, dim, inter * 3 // 2, VOCAB, chunk)
    new = lambda: rx.build_synthetic(cfg, dev, max_slots=slots, max_context=prompt + 192)
    qcfg = qh.QwenHybridConfig(vocab_size=VOCAB, hidden_size=width, intermediate_size=inter, num_hidden_layers=LAYERS,
                               num_attention_heads=heads, num_key_value_heads=kv, attn_output_gate=False,
                               layer_types=["full_attention"] * LAYERS)
    old = lambda: qh.build_synthetic(qcfg, dev, max_slots=slots, max_context=prompt + 192)
    return new, old


def _throughput(make, dev, prompt: int, slots: int, timer: _Timer) -> dict:
    rt = make()
    gen = torch.Generator().manual_seed(1)
    ids = torch.randint(0, VOCAB, (prompt,), generator=gen, dtype=torch.int32).to(dev)
    slot = rt.allocate()

    def prefill():
        nonlocal slot
        rt.free(slot)
        slot = rt.allocate()
        rt.prefill(slot, ids, prompt)
    out = {"prefill_tok_s": round(prompt / timer(prefill) * 1e3, 0)}
    slots_l = [slot]
    while len(slots_l) < slots:
        s = rt.allocate()
        rt.prefill(s, ids, prompt)
        slots_l.append(s)
    for b in (1, slots):
        tok = torch.ones(b, dtype=torch.int32, device=dev)
        ms = timer(lambda: rt.decode(slots_l[:b], tok))
        out[f"decode_b{b}_tok_s"] = round(b / ms * 1e3, 1)
        out[f"decode_b{b}_ms"] = round(ms, 4)
    return out


def _recorder(timer: _Timer):
    """(rows, pair): ``pair(what, shape, new, like)`` times two (call, bytes, flops) and appends one row: ms and roofline
    fraction of both and the distance ratio."""
    peaks, _ = _peaks()
    bw, fl = peaks["hbm_gbs"] * 1e6, peaks["bf16_tflops"] * 1e9            # bytes, flops per ms
    rows_out: list[dict] = []

    def pair(what, shape, new, old):
        rec, frac = {"kernel": what, "shape": shape}, {}
        for tag, spec in (("new", new), ("like", old)):
            if spec is None:
                continue
            fn, need_bytes, need_flops = spec
            ms = timer(fn)
            roof = max(need_bytes / bw, need_flops / fl)
            frac[tag] = roof / ms
            rec[tag] = {"ms": round(ms, 4), "fraction": round(roof / ms, 3), "bound": "memory" if need_bytes / bw >= need_flops / fl else "tensor"}
        if "like" in rec:
            rec["distance_ratio"] = round(frac["like"] / frac["new"], 2)
        rows_out.append(rec)
    return rows_out, pair


def _kernels(size: str, dev, timer: _Timer, ctx: int) -> list[dict]:
    """One row per kernel pair: (what, shape, new ms and fraction, like kernel ms and fraction)."""
    from ..ops import attention, basic, gemm, mixattn
    from ..models import rutulix as rx
    width, H, G, D, inter, chunk = SIZES[size]
    ff = inter * 3 // 2
    rnd = lambda *s, dt=torch.bfloat16: torch.randn(*s, device=dev, dtype=torch.float32).to(dt)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    cfg = rx.RutulixConfig.uniform(1, width, H, G, D, ff, 64, chunk)
    m = rx.RutulixWeights(cfg, rx.synth_state(cfg, 0, dev), dev).layers[0].mix
    rows_out, pair = _recorder(timer)
    bs, pages = 64, (ctx + 63) // 64
    for t in (8192, 32):
        x32, x16, d16 = rnd(t, width, dt=torch.float32), rnd(t, width), rnd(t, width)
        g32, g16 = torch.ones(width, device=dev), torch.ones(width, device=dev, dtype=torch.bfloat16)
        # fp32 residual read + written, delta read, output written against a bf16 residual
        pair("residual + norms", f"{t} x {width}",
             (lambda: mixattn.residual_norm(x32, width, 1e-5, delta=d16, bias=g32, post_w=g32, pre_w=g32), t * width * 12, 0),
             (lambda: basic.add_rmsnorm(x16, d16, g16, 1e-5), t * width * 8, 0))
        z, gu = rnd(t, ff), rnd(t, 2 * inter)
        bias = torch.ones(ff, device=dev)
        pair("activation on its own", f"{t} x {ff}", (lambda: mixattn.bias_xielu(z, bias, 0.7, 1.2), t * ff * 4, 0),
             (lambda: basic.silu_mul(gu), t * inter * 6, 0))
        # attention prologue
        proj, qkv = rnd(t, (H + G) * D), rnd(t, (H + 2 * G) * D)
        kc, vc = (torch.zeros(max(t, 64) // bs + 1, bs, G * D, dtype=torch.bfloat16, device=dev) for _ in range(2))
        k4, v4 = (torch.zeros(max(t, 64) // bs + 1, G, bs, D, dtype=torch.bfloat16, device=dev) for _ in range(2))
        pos, qn = torch.arange(t, dtype=torch.int32, device=dev), torch.ones(D, device=dev, dtype=torch.bfloat16)
        inv = attention.rope_inv_freq(m.rot, 5e5, dev)
        n_mix = t if t > 32 else 0
        qout = t * H * (G * D * 2 if n_mix else D * 4)
        pair("attention prologue", f"{t} tokens", (lambda: mixattn.qk_row_prep(proj, m, pos, pos, kc, vc, n_mix),
                                                   t * (H + G) * D * 2 + t * 2 * G * D * 2 + qout, 0),
             (lambda: attention.qk_norm_rope_append(qkv, 0, D, False, qkv, H * D, qkv, (H + G) * D, qn, qn, True, 1e-5, inv, m.rot,
                                                    pos, pos, k4, v4, H, G), t * (H + 2 * G) * D * 2 * 2, 0))
    # prompt attention: one chunk-aligned prompt
    t = 8192
    table = (torch.arange(t // bs, dtype=torch.int32, device=dev) + 1)[None]
    q_mix, q = rnd(t, H, G * D), rnd(t, H, D)
    kc, vc = (rnd(t // bs + 1, bs, G * D) for _ in range(2))
    k4, v4 = kc.view(-1, G, bs, D), vc.view(-1, G, bs, D)
    out = torch.empty(t, H * D, dtype=torch.bfloat16, device=dev)
    pairs_n = sum((p % chunk + 1) for p in range(t))
    full_n = t * (t + 1) // 2
    args = (i32([0]), i32([t]), i32([t]), t)
    new_fn = lambda: mixattn.prefill(q_mix, m, kc, vc, table, *args, out)
    old_fn = lambda: attention.prefill(q, k4, v4, table, *args)
    pair("prompt attention (multiplications executed)", f"{t} tokens, chunk {chunk}",
         (new_fn, 0, 2 * pairs_n * H * (G * D + D)), (old_fn, 0, 2 * full_n * H * 2 * D))
    pair("prompt attention (mixing counted as H x H per pair)", f"{t} tokens, chunk {chunk}",
         (new_fn, 0, 2 * pairs_n * H * (2 * D + H)), (old_fn, 0, 2 * full_n * H * 2 * D))
    # decode attention
    for b in (1, 32):
        keys = min(ctx, chunk)
        tb = (torch.arange(b * pages, dtype=torch.int32, device=dev) + 1).view(b, pages)
        kc, vc = (rnd(b * pages + 1, bs, G * D) for _ in range(2))
        k4, v4 = kc.view(-1, G, bs, D), vc.view(-1, G, bs, D)
        qr, q = rnd(b, H, D, dt=torch.float32), rnd(b, H, D)
        ob = torch.empty(b, H * D, dtype=torch.bfloat16, device=dev)
        pos, kvl = i32([keys - 1] * b), i32([keys] * b)
        nbytes = b * keys * G * D * 2 * 2
        pair("decode attention", f"batch {b}, {keys} keys", (lambda: mixattn.rows(qr, m, kc, vc, tb, pos, keys, ob), nbytes, 0),
             (lambda: attention.decode(q, k4, v4, tb, kvl, max_kv_len=keys), nbytes, 0))
    # projections: the up projection with bias + activation in its epilogue beside the plain product of the same GEMM
    for t in (8192, 32):
        w, x, bias = gemm.PackedLinear.from_bf16(rnd(ff, width)), rnd(t, width), torch.ones(ff, device=dev)
        need = ((ff * width + t * width + t * ff) * 2, 2 * t * ff * width)
        pair("up projection + bias + activation (like: plain product)", f"{t} x {ff} x {width}",
             (lambda: gemm.linear_bias_xielu(x, w, bias, 0.7, 1.2), *need), (lambda: gemm.linear(x, w), *need))
        n = (H + G) * D
        wq = gemm.PackedLinear.from_bf16(rnd(n, width))
        pair("q | k projection", f"{t} x {n} x {width}",
             (lambda: gemm.linear(x, wq), (n * width + t * width + t * n) * 2, 2 * t * n * width), None)
    return rows_out


def _zg_models(size: str, dev, prompt: int, slots: int):
    from ..models import qwen_hybrid as qh
    from ..models import zigasun as zg
    width, heads, kv, dim, vdim, ff, inner, states, rank = ZG_SIZES[size]
    cfg = zg.ZigasunConfig.alternating(LAYERS, width, heads, kv, dim, vdim, ff, inner, states, rank, VOCAB)
    for L in cfg.layers:                       # the closest model has a feed-forward in every layer
        L.ff, L.limit = ff, 7.0
    new = lambda: zg.build_synthetic(cfg, dev, max_slots=slots, max_context=prompt + 192)
    qcfg = qh.QwenHybridConfig(vocab_size=VOCAB, hidden_size=width, intermediate_size=ff, num_hidden_layers=LAYERS,
                               num_attention_heads=heads, num_key_value_heads=kv, attn_output_gate=False,
                               linear_num_key_heads=16, linear_num_value_heads=inner // 128,
                               layer_types=["full_attention", "linear_attention"] * (LAYERS // 2))
    old = lambda: qh.build_synthetic(qcfg, dev, max_slots=slots, max_context=prompt + 192)
    return new, old


def _zg_kernels(size: str, dev, timer: _Timer, ctx: int) -> list[dict]:
    from ..models import zigasun as zg
    from ..ops import attention, basic, decoder, diffattn, gdn, gemm, scan
    width, H, G, D, V, ff, inner, N, rank = ZG_SIZES[size]
    rnd = lambda *s, dt=torch.bfloat16: torch.randn(*s, device=dev, dtype=torch.float32).to(dt)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    cfg = zg.ZigasunConfig.alternating(2, width, H, G, D, V, ff, inner, N, rank, 64)
    w = zg.ZigasunWeights(cfg, zg.synth_state(cfg, 0, dev), dev)
    aw, sw = w.layers[0].mix, w.layers[1].mix
    m = aw.m
    rows_out, pair = _recorder(timer)
    bs, pages = 64, (ctx + 63) // 64
    hv, hk = inner // 128, 16
    for t in (8192, 32):
        x32, x16, d16 = rnd(t, width, dt=torch.float32), rnd(t, width), rnd(t, width)
        g32, g16 = torch.ones(width, device=dev), torch.ones(width, device=dev, dtype=torch.bfloat16)
        # fp32 residual read + written, delta read, output written against a bf16 residual
        pair("residual + norm", f"{t} x {width}",
             (lambda: decoder.residual_norm(x32, width, 1e-5, delta=d16, post_w=g32, rms=True, plain=True), t * width * 12, 0),
             (lambda: basic.add_rmsnorm(x16, d16, g16, 1e-5), t * width * 8, 0))
        gu = rnd(t, 2 * ff)
        pair("gated unit on its own", f"{t} x {ff}", (lambda: decoder.glu(gu, decoder.GLU_TILE, 7.0), t * ff * 6, 0),
             (lambda: basic.silu_mul(gu), t * ff * 6, 0))
        proj, qkv = rnd(t, aw.proj.n), rnd(t, (H + 2 * G) * 128)
        kc, vc = (torch.zeros(max(t, 64) // bs + 1, bs, n, dtype=torch.bfloat16, device=dev) for n in (m.k_width, m.v_width))
        k4, v4 = (torch.zeros(max(t, 64) // bs + 1, G, bs, 128, dtype=torch.bfloat16, device=dev) for _ in range(2))
        pos, qn = torch.arange(t, dtype=torch.int32, device=dev), torch.ones(128, device=dev, dtype=torch.bfloat16)
        inv = attention.rope_inv_freq(64, 5e5, dev)
        pair("attention prologue", f"{t} tokens",
             (lambda: diffattn.head_prep(proj, m, pos, pos, kc, vc), t * (m.q_width + m.k_width + m.v_width) * 4, 0),
             (lambda: attention.qk_norm_rope_append(qkv, 0, 128, False, qkv, H * 128, qkv, (H + G) * 128, qn, qn, True, 1e-5, inv, 64,
                                                    pos, pos, k4, v4, H, G), t * (H + 2 * G) * 128 * 4, 0))
        # up projection with the gated unit (epilogue of the pair GEMM, or a second kernel) beside the plain product
        wu, xs = decoder.Projection.make(rnd(2 * ff, width), torch.bfloat16, dev), rnd(t, width)
        need = ((2 * ff * width + t * width + t * ff) * 2, 2 * t * 2 * ff * width)
        plain = ((2 * ff * width + t * width + 2 * t * ff) * 2, 2 * t * 2 * ff * width)
        pair("gate | up projection + gated unit (like: plain product)", f"{t} x {2 * ff} x {width}",
             (lambda: wu.glu(xs, 7.0), *need), (lambda: gemm.linear(xs, wu.packed), *plain))
        for what, pr, o32 in (("q | k | v | g projection (like: none)", aw.proj, False), ("B | C | dt projection (like: none)", sw.x, False),
                              ("step size projection (like: none)", sw.dt, True)):
            xk = rnd(t, pr.k)
            pair(what, f"{t} x {pr.n} x {pr.k}", (lambda: pr(xk, out_f32=o32), (pr.n * pr.k + t * pr.k) * 2 + t * pr.n * (4 if o32 else 2),
                                                  2 * t * pr.n * pr.k), None)
        # convolution
        xin, cw = rnd(t, 2 * inner), rnd(inner, 4)
        tails = torch.zeros(t if t <= 32 else 1, 3, inner, dtype=torch.bfloat16, device=dev)
        ar, one, zero = torch.arange(t, dtype=torch.int32, device=dev), torch.ones(t, dtype=torch.int32, device=dev), torch.zeros(t, dtype=torch.int32, device=dev)
        seg = scan.Segments(ar, ar, ar, one, ar, 1) if t <= 32 else scan.Segments(zero, zero, i32([0]), i32([t]), i32([0]), t)
        pos1 = ar + 5
        like_conv = (lambda: basic.conv_silu_step(xin[:, :inner], cw, tails, ar)) if t <= 32 else (lambda: basic.conv_silu(xin[:, :inner], cw, tails[0]))
        cbytes = t * inner * 4 + (t * 3 * inner * 2 if t <= 32 else 0)
        pair("convolution", f"{t} x {inner}", (lambda: scan.conv_rows(xin[:, :inner], sw.conv, sw.conv_b, tails, seg, pos1), cbytes, 0),
             (like_conv, cbytes, 0))
        # recurrence: rows in and out, state read and written once per sequence
        xc, dt, bc = rnd(t, inner), rnd(t, inner, dt=torch.float32), rnd(t, sw.x.n)
        n_seq = seg.first.numel()
        st = torch.zeros(n_seq, inner, N, dtype=torch.float32, device=dev)
        sbytes = t * inner * 10 + t * sw.x.n * 2 + n_seq * inner * N * 8
        mixed, gg = rnd(t, (2 * hk + hv) * 128), -torch.rand(t, hv, device=dev)
        beta = torch.rand(t, hv, device=dev)
        gst = torch.zeros(n_seq, hv, 128, 128, dtype=torch.float32, device=dev)
        gbytes = t * (2 * hk + 2 * hv) * 256 + t * hv * 8 + n_seq * hv * 128 * 128 * 8
        like = (lambda: gdn.step(gst, ar, mixed, 0, hk * 128, 2 * hk * 128, gg, beta, hv, hk)) if t <= 32 else \
            (lambda: gdn.chunked(mixed, 0, hk * 128, 2 * hk * 128, gg, beta, gst[0], hv, hk))
        pair("recurrence", f"{t} tokens, {inner} channels x {N} states",
             (lambda: scan.selective_scan(xc, dt, bc, sw.b_off, sw.c_off, xin[:, inner:], sw.a, sw.dt_b, sw.d, st, seg, pos1, xin[:, :inner], tails), sbytes, 0),
             (like, gbytes, 0))
    # decoding step with as much state as the like kernel holds for 32 sequences
    t = 32 * 128 // N
    xc, dt, bc, xin = rnd(t, inner), rnd(t, inner, dt=torch.float32), rnd(t, sw.x.n), rnd(t, 2 * inner)
    ar, one = torch.arange(t, dtype=torch.int32, device=dev), torch.ones(t, dtype=torch.int32, device=dev)
    seg, pos1, st = scan.Segments(ar, ar, ar, one, ar, 1), ar + 5, torch.zeros(t, inner, N, dtype=torch.float32, device=dev)
    mixed, gg, beta = rnd(32, (2 * hk + hv) * 128), -torch.rand(32, hv, device=dev), torch.rand(32, hv, device=dev)
    gst = torch.zeros(32, hv, 128, 128, dtype=torch.float32, device=dev)
    pair("recurrence, equal state bytes", f"{t} sequences (like: 32), {inner} channels x {N} states",
         (lambda: scan.selective_scan(xc, dt, bc, sw.b_off, sw.c_off, xin[:, inner:], sw.a, sw.dt_b, sw.d, st, seg, pos1),
          t * inner * 10 + t * sw.x.n * 2 + t * inner * N * 8, 0),
         (lambda: gdn.step(gst, ar[:32], mixed, 0, hk * 128, 2 * hk * 128, gg, beta, hv, hk),
          32 * (2 * hk + 2 * hv) * 256 + 32 * hv * 8 + 32 * hv * 128 * 128 * 8, 0))
    t = 8192
    table = (torch.arange(t // bs, dtype=torch.int32, device=dev) + 1)[None]
    q, q1 = rnd(t, H, 2, D), rnd(t, H, 128)
    kc, vc = rnd(t // bs + 1, bs, m.k_width), rnd(t // bs + 1, bs, m.v_width)
    k4, v4 = (rnd(t // bs + 1, G, bs, 128) for _ in range(2))
    out, gate = torch.empty(t, H * V, dtype=torch.bfloat16, device=dev), rnd(t, H)
    full_n = t * (t + 1) // 2
    args = (i32([0]), i32([t]), i32([t]), t)
    pair("prompt attention", f"{t} tokens", (lambda: diffattn.prefill(q, m, kc, vc, gate, table, *args, out), 0, 2 * full_n * H * 2 * (D + V)),
         (lambda: attention.prefill(q1, k4, v4, table, *args), 0, 2 * full_n * H * 2 * 128))
    for b in (1, 32):
        tb = (torch.arange(b * pages, dtype=torch.int32, device=dev) + 1).view(b, pages)
        kc, vc = rnd(b * pages + 1, bs, m.k_width), rnd(b * pages + 1, bs, m.v_width)
        k4, v4 = (rnd(b * pages + 1, G, bs, 128) for _ in range(2))
        q, q1, gate = rnd(b, H, 2, D), rnd(b, H, 128), rnd(b, H)
        ob = torch.empty(b, H * V, dtype=torch.bfloat16, device=dev)
        pos, kvl = i32([ctx - 1] * b), i32([ctx] * b)
        pair("decode attention", f"batch {b}, {ctx} keys", (lambda: diffattn.rows(q, m, kc, vc, gate, tb, pos, ctx, ob), b * ctx * (m.k_width + m.v_width) * 2, 0),
             (lambda: attention.decode(q1, k4, v4, tb, kvl, max_kv_len=ctx), b * ctx * G * 128 * 4, 0))
    return rows_out


def _kx_models(size: str, dev, prompt: int, slots: int):
    from ..models import kemirax as kx
    from ..models import mla_moe as mm
    from ..models import mla_moe_gpu as mg
    width, H, d, r, v, qr, c, gh, ff, E, ident, top = KX_SIZES[size]
    cfg = kx.KemiraxConfig.pattern(KX_LAYERS, width, H, d, r, v, qr, c, gh, 128, 128, ff, E, ident, top, ff, VOCAB)
    new = lambda: kx.build_synthetic(cfg, dev, max_slots=slots, max_context=prompt + 192)
    mcfg = mm.MlaMoeConfig(vocab_size=VOCAB, hidden_size=width, num_layers=len(KX_LAYERS), first_dense_layers=0, q_lora_rank=qr,
                           kv_lora_rank=c, num_heads=H, qk_nope_dim=d, qk_rope_dim=r, v_head_dim=v, index_heads=0, index_dim=0,
                           index_topk=0, num_experts=E, experts_per_token=top, num_shared_experts=1, expert_intermediate=ff,
                           score_func="softmax", route_scale=1.0, norm_topk=False, expert_format="bf16")
    old = lambda: mg.MlaMoeBatchRuntime(mcfg, mg.MlaMoeGpuWeights(mcfg, mm.synth_state(mcfg, 0, dev), dev), max_slots=slots,
                                        max_context=prompt + 192)
    return new, old


def _kx_kernels(size: str, dev, timer: _Timer, ctx: int) -> list[dict]:
    from ..models import kemirax as kx
    from ..ops import basic, decoder, gdn, gemm, gla, latent, mla, moe, scan
    width, H, d, r, v, qr, c, gh, ff, E, ident, top = KX_SIZES[size]
    rnd = lambda *s, dt=torch.bfloat16: torch.randn(*s, device=dev, dtype=torch.float32).to(dt)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    cfg = kx.KemiraxConfig.pattern("ag", width, H, d, r, v, qr, c, gh, 128, 128, ff, E, ident, top, ff, 64)
    w = kx.KemiraxWeights(cfg, kx.synth_state(cfg, 0, dev), dev)
    lay, aw, gw, ew = w.layers[0], w.layers[0].mix, w.layers[1].mix, w.layers[0].ff
    m, gm = aw.m, gw.m
    rows_out, pair = _recorder(timer)
    bs, pages, cw = 64, (ctx + 63) // 64, c + r
    for t in (8192, 32):
        ar, one, zero = torch.arange(t, dtype=torch.int32, device=dev), torch.ones(t, dtype=torch.int32, device=dev), torch.zeros(t, dtype=torch.int32, device=dev)
        seg = scan.Segments(ar, ar, ar, one, ar, 1) if t <= 32 else scan.Segments(zero, zero, i32([0]), i32([t]), i32([0]), t)
        n_seq, pos1 = seg.first.numel(), ar + 5
        # ---- step between the layers: everything the residual takes, beside the plain residual add + norm
        x32, x16, h16, d16 = rnd(t, width, dt=torch.float32), rnd(t, width), rnd(t, width), rnd(t, width)
        xo, g16 = torch.empty_like(x32), torch.ones(width, device=dev, dtype=torch.bfloat16)
        z = moe.router_logits(h16, ew.router)
        idx, wts = moe.route(z[:, :E + ident], ew.correction, top, "softmax", False, 1.0)
        y, row = moe.experts_rows(h16, idx, ew.w13, ew.w2, 0, 7.0, kx.UNIT_SLOPE)
        gates, tails = lay.gates(h16), torch.zeros(max(n_seq, 1), width, dtype=torch.bfloat16, device=dev)
        local = int((idx < E).sum())
        args = dict(ld=width, n=t, dtype=torch.bfloat16, x_out=xo, mix=d16, gates=gates, gate_b=lay.gate_b, h=h16,
                    routed=decoder.Routed(y, row, idx, wts, E), shared=x16, shared_gate=z[:, E + ident:], shift=lay.shift, tail=tails,
                    seg=seg, positions=pos1)
        pair("step between layers (gates, experts' sum, residual, norm, shift; like: residual + norm)", f"{t} x {width}",
             (lambda: decoder.parallel_step(x32, width, 1.0, 1e-5, **args), t * width * (8 + 2 + 4 + 2 + 2 + 2 + 2) + local * width * 2, 0),
             (lambda: basic.add_rmsnorm(x16, d16, g16, 1e-5), t * width * 8, 0))
        # ---- experts: routing, plan, gather, both products, unit; beside the same with SwiGLU and the combine
        each = 3 * width * ff * 2
        ebytes = int(torch.unique(idx[idx < E]).numel()) * each              # experts that have a token
        need = (ebytes + t * width * 2 + local * width * 2, 2 * local * 3 * width * ff)
        i2, w2_ = moe.route(z[:, :E], None, top, "softmax", False, 1.0)
        ebytes2 = int(torch.unique(i2).numel()) * each
        pair("routed experts (like: with SwiGLU and combine)", f"{t} tokens, {top} of {E}",
             (lambda: moe.experts_rows(h16, idx, ew.w13, ew.w2, 0, 7.0, kx.UNIT_SLOPE), *need),
             (lambda: moe.experts_forward(h16, i2, w2_, ew.w13, ew.w2, 0), ebytes2 + t * width * 4, 2 * t * top * 3 * width * ff))
        pair("routing (like: sigmoid, normalised)", f"{t} x {E + ident}",
             (lambda: moe.route(z[:, :E + ident], ew.correction, top, "softmax", False, 1.0), t * (z.stride(0) * 4 + top * 8), 0),
             (lambda: moe.route(z[:, :E], ew.correction[:E], top, "sigmoid", True, 1.0), t * (z.stride(0) * 4 + top * 8), 0))
        # ---- latent attention around the attention itself
        proj, q = rnd(t, aw.down.n), rnd(t, aw.uq.n)
        cache = torch.zeros(max(t, 64) // bs + 1, bs, cw, dtype=torch.bfloat16, device=dev)
        kvp, gam, qn = rnd(t, cw), torch.ones(c, device=dev, dtype=torch.bfloat16), rnd(t, qr)
        gq = torch.ones(qr, device=dev, dtype=torch.bfloat16)
        pair("latent prologue (like: query norm, cache append)", f"{t} tokens",
             (lambda: latent.prep(proj, m, pos1, ar, cache), t * (qr + cw) * 4, 0),
             (lambda: (basic.rmsnorm(qn, gq, 1e-5), mla.kv_append(kvp, gam, 1e-5, pos1, ar, 1e4, cache.view(-1, cw), c, r)), t * (qr + cw) * 4, 0))
        if t > 32:
            qs = torch.empty(t, H * (d + r), dtype=torch.bfloat16, device=dev)
            pair("query rotation (like: split and rotate)", f"{t} tokens", (lambda: latent.rotate_heads(q, m, pos1), t * H * r * 4, 0),
                 (lambda: mla.q_prepare(qs, pos1, 1e4, H, d, r), t * H * (d + r) * 4, 0))
        else:
            qa, ol = torch.empty(t, H, cw, dtype=torch.bfloat16, device=dev), rnd(t, H, c)
            qh, oh, out = rnd(H, t, d), rnd(H, t, c), torch.empty(t, H * v, dtype=torch.bfloat16, device=dev)
            wk = aw.uk.reshape(H * c, d)
            pair("queries to the latent space", f"{t} tokens",
                 (lambda: latent.head_linear(q, q.stride(0), d + r, aw.uk, qa, qa.stride(0), cw, t), (H * c * d + t * H * (d + c)) * 2, 2 * t * H * c * d),
                 (lambda: mla.per_head_linear(qh, wk), (H * c * d + t * H * (d + c)) * 2, 2 * t * H * c * d))
            wv = aw.uv.reshape(H * v, c)
            pair("latents to values (like: with the transpose)", f"{t} tokens",
                 (lambda: latent.head_linear(ol, ol.stride(0), c, aw.uv, out, out.stride(0), v, t), (H * v * c + t * H * (v + c)) * 2, 2 * t * H * c * v),
                 (lambda: mla.transpose_heads(mla.per_head_linear(oh, wv)), (H * v * c + t * H * (v + c)) * 2, 2 * t * H * c * v))
        # ---- recurrence: rows in and out, state read and written once per sequence
        gp, st = rnd(t, gw.proj.n), torch.zeros(n_seq, gh, 128, 128, dtype=torch.float32, device=dev)
        sbytes = t * (gh * 128 * 5 + gm.rank) * 2 + n_seq * gh * 128 * 128 * 8
        mixed, gg = rnd(t, 3 * gh * 128), -torch.rand(t, gh, device=dev)
        beta, gate = torch.rand(t, gh, device=dev), rnd(t * gh, 128)
        gst = torch.zeros(n_seq, gh, 128, 128, dtype=torch.float32, device=dev)
        nw = torch.ones(128, dtype=torch.bfloat16, device=dev)
        like = (lambda: gdn.step(gst, ar, mixed, 0, gh * 128, 2 * gh * 128, gg, beta, gh, gh)) if t <= 32 else \
            (lambda: gdn.chunked(mixed, 0, gh * 128, 2 * gh * 128, gg, beta, gst[0], gh, gh))
        pair("recurrence with decay, norm and gate (like: Gated DeltaNet, gated norm)", f"{t} tokens, {gh} heads x 128 x 128",
             (lambda: gla.recurrence(gp, gm, st, seg, pos1, gw.o.k), sbytes, 0),
             (lambda: basic.gated_rmsnorm(like().view(t * gh, 128), gate, nw), sbytes, 0))
    # ---- prompt attention, whole prompt: the products a pair needs with keys and values expanded; expansion included below
    t = 8192
    table = (torch.arange(t // bs, dtype=torch.int32, device=dev) + 1)[None]
    cache, q, ql, qp = rnd(t // bs + 1, bs, cw), rnd(t, aw.uq.n), rnd(H, t, c), rnd(t, H, r)
    out = torch.empty(t, H * v, dtype=torch.bfloat16, device=dev)
    e0, et, pos = i32([0]), i32([t]), torch.arange(t, dtype=torch.int32, device=dev)
    full = t * (t + 1) // 2
    flops, absorbed = 2 * full * H * (d + r + v), 2 * full * H * (2 * c + r)
    lat, key = latent.gather(cache, m, table, e0, et, e0, t)
    kv = gemm.linear(lat, aw.ukv)
    L, _lib, ptr = latent._lib.lib(), latent._lib, latent._lib.ptr
    tiles = lambda: _lib.check(L.b200_attn_heads_prefill(
        ptr(q), q.stride(0), ptr(kv), ptr(key), key.shape[1], ptr(out), out.stride(0), ptr(e0), ptr(et), ptr(et), ptr(e0), 1, t, t,
        lat.shape[0], 0, H, m.d, m.r, m.v, latent._f(m.scale), ptr(_lib.status_word(dev)), _lib.stream()), "attn_heads_prefill")
    like = lambda: mla.attention(ql, qp, cache.view(-1, cw), table, bs, pos, c, r, m.scale, max_keys=t)
    pair("prompt attention, products executed (like: absorbed)", f"{t} tokens", (tiles, 0, flops), (like, 0, absorbed))
    pair("prompt attention with expansion, expanded products counted for both", f"{t} tokens",
         (lambda: latent.attend_tiles(q, m, *latent.gather(cache, m, table, e0, et, e0, t), aw.ukv, e0, et, et, e0, t, out), 0,
          flops + 2 * t * H * c * (d + v)), (like, 0, flops))
    for b in (1, 32):
        tb = (torch.arange(b * pages, dtype=torch.int32, device=dev) + 1).view(b, pages)
        cache = rnd(b * pages + 1, bs, cw)
        qa, ql, qp, pos = rnd(b, H, cw), rnd(H, b, c), rnd(b, H, r), i32([ctx - 1] * b)
        seq = torch.arange(b, dtype=torch.int32, device=dev)
        need = (b * ctx * cw * 2, 2 * b * ctx * H * (2 * c + r))
        pair("decode attention", f"batch {b}, {ctx} keys", (lambda: latent.attend_rows(qa, m, cache, tb, pos, ctx), *need),
             (lambda: mla.attention(ql, qp, cache.view(-1, cw), tb, bs, pos, c, r, m.scale, seq_of_token=seq, max_keys=ctx), *need))
    return rows_out


def _ns_config(size: str, kinds: str, vocab: int):
    from ..models import nunosun as ns
    width, H, G, window, rh, dh, dg, inter, E, top, side = NS_SIZES[size]
    return ns.NunosunConfig.pattern(kinds, width, H, G, 128, 128, window, rh, 128, 128, dh, dg, 128, 128, inter * 3 // 2, inter // top, E, top,
                                    side, vocab)


def _ns_models(size: str, dev, prompt: int, slots: int):
    from ..models import nunosun as ns
    from ..models import qwen_hybrid as qh
    width, H, G, _, _, dh, dg, inter, *_ = NS_SIZES[size]
    cfg = _ns_config(size, NS_LAYERS, VOCAB)
    new = lambda: ns.build_synthetic(cfg, dev, max_slots=slots, max_context=prompt + 192)
    qcfg = qh.QwenHybridConfig(vocab_size=VOCAB, hidden_size=width, intermediate_size=inter, num_hidden_layers=LAYERS,
                               num_attention_heads=H, num_key_value_heads=G, attn_output_gate=False, linear_num_key_heads=dg,
                               linear_num_value_heads=dh, layer_types=["linear_attention", "full_attention"] * (LAYERS // 2))
    old = lambda: qh.build_synthetic(qcfg, dev, max_slots=slots, max_context=prompt + 192)
    return new, old


def _ns_kernels(size: str, dev, timer: _Timer, ctx: int) -> list[dict]:
    from ..models import nunosun as ns
    from ..ops import attention, basic, decay, decoder, gdn, gemm, moe, scan, winattn
    width, H, G, window, rh, dh, dg, inter, E, top, side = NS_SIZES[size]
    ff, eff = inter * 3 // 2, inter // top
    rnd = lambda *s, dt=torch.bfloat16: torch.randn(*s, device=dev, dtype=torch.float32).to(dt)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    cfg = _ns_config(size, "dp", 64)
    w = ns.NunosunWeights(cfg, ns.synth_state(cfg, 0, dev), dev)
    dl, pl = w.layers
    dw, pw, ew, dense = dl.mix, pl.mix, pl.ff, dl.ff
    m = pw.left
    rows_out, pair = _recorder(timer)
    bs, pages = 64, (ctx + 63) // 64
    for t in (8192, 32):
        ar, one, zero = torch.arange(t, dtype=torch.int32, device=dev), torch.ones(t, dtype=torch.int32, device=dev), torch.zeros(t, dtype=torch.int32, device=dev)
        seg = scan.Segments(ar, ar, ar, one, ar, 1) if t <= 32 else scan.Segments(zero, zero, i32([0]), i32([t]), i32([0]), t)
        n_seq, pos1 = seg.first.numel(), ar + 5
        # ---- the two residual steps of a layer, beside the plain residual add + norm
        x32, x16, h16, d16 = rnd(t, width, dt=torch.float32), rnd(t, width), rnd(t, width), rnd(t, width)
        xo, g16 = torch.empty_like(x32), torch.ones(width, device=dev, dtype=torch.bfloat16)
        z = moe.router_logits(h16, ew.router)[:, :E]
        idx, wts = moe.route(z, ew.router_b, top, "softmax_chosen", True, 1.0)
        y, row = moe.experts_rows(h16, idx, ew.w13, ew.w2)
        common = dict(ld=width, n=t, dtype=torch.bfloat16, x_out=xo)
        like_step = (lambda: basic.add_rmsnorm(x16, d16, g16, 1e-5), t * width * 8, 0)
        pair("step behind the pair and the experts (like: residual + norm)", f"{t} x {width}",
             (lambda: decoder.branch_step(x32, width, 1e-5, normed=((d16, pw.left_w), (x16, pw.right_w)),
                                          routed=decoder.Routed(y, row, idx, wts, E), copy=True, **common), t * width * (8 + 4 + 2 + 2 * top), 0),
             like_step)
        pair("step behind the delta rule and the dense unit (like: residual + norm)", f"{t} x {width}",
             (lambda: decoder.branch_step(x32, width, 1e-5, plain=(d16, x16), copy=True, **common), t * width * (8 + 4 + 2), 0), like_step)
        tails = torch.zeros(n_seq, 3, width, dtype=torch.bfloat16, device=dev)
        pair("step in front of a layer, with the row convolution (like: residual + norm)", f"{t} x {width}",
             (lambda: decoder.branch_step(x32, width, 1e-5, normed=((d16, dl.side_norm),), weight=dl.norm, conv=dl.conv, tail=tails, seg=seg,
                                          positions=pos1, **common), t * width * (8 + 2 + 2 + (4 if t > 32 else 2)), 0), like_step)
        # ---- activations and the side input
        zu, gu = rnd(t, ff), rnd(t, 2 * inter)
        pair("polynomial of row norms (like: SwiGLU unit)", f"{t} x {ff}", (lambda: decoder.poly_norm(zu, ff, dense.act, 1e-5, ff), t * ff * 4, 0),
             (lambda: basic.silu_mul(gu), t * inter * 6, 0))
        ids, wg = ar % 64, gemm.PackedLinear.from_bf16(rnd(2 * side, width))
        pair("side gate with its projection (like: SwiGLU unit with its projection)", f"{t} x {side} x {width}",
             (lambda: decoder.token_gate(h16, dl.side_gate, w.side_embed, 0, ids), (side * width + t * width + 2 * t * side) * 2, 2 * t * side * width),
             (lambda: basic.silu_mul(gemm.linear(h16, wg)), (2 * side * width + t * width + t * side) * 2, 4 * t * side * width))
        # ---- experts
        each = 3 * width * eff * 2
        ebytes = int(torch.unique(idx).numel()) * each
        i2, w2_ = moe.route(z, None, top, "softmax", False, 1.0)
        ebytes2 = int(torch.unique(i2).numel()) * each
        pair("routed experts (like: with combine)", f"{t} tokens, {top} of {E}",
             (lambda: moe.experts_rows(h16, idx, ew.w13, ew.w2), ebytes + t * width * 2 * (1 + top), 2 * t * top * 3 * width * eff),
             (lambda: moe.experts_forward(h16, i2, w2_, ew.w13, ew.w2, 0), ebytes2 + t * width * 4, 2 * t * top * 3 * width * eff))
        pair("routing (like: sigmoid, normalised)", f"{t} x {E}",
             (lambda: moe.route(z, ew.router_b, top, "softmax_chosen", True, 1.0), t * (z.stride(0) * 4 + top * 8), 0),
             (lambda: moe.route(z, ew.router_b, top, "sigmoid", True, 1.0), t * (z.stride(0) * 4 + top * 8), 0))
        # ---- attention prologue
        proj, qkv = rnd(t, pw.proj.n), rnd(t, (H + 2 * G) * 128)
        kc, vc = (torch.zeros(max(t, 64) // bs + 1, bs, G * 128, dtype=torch.bfloat16, device=dev) for _ in range(2))
        k4, v4 = (torch.zeros(max(t, 64) // bs + 1, G, bs, 128, dtype=torch.bfloat16, device=dev) for _ in range(2))
        qn, inv = torch.ones(128, device=dev, dtype=torch.bfloat16), attention.rope_inv_freq(64, 5e5, dev)
        nb = t * (H + 2 * G) * 128 * 4
        pair("attention prologue", f"{t} tokens", (lambda: winattn.head_prep(proj, m, ar, ar, kc, vc), nb, 0),
             (lambda: attention.qk_norm_rope_append(qkv, 0, 128, False, qkv, H * 128, qkv, (H + G) * 128, qn, qn, True, 1e-5, inv, 64,
                                                    ar, ar, k4, v4, H, G), nb, 0))
        # ---- recurrences: projected rows in, gated rows out, state read and written once per sequence
        dp, st = rnd(t, dw.proj.n), torch.zeros(n_seq, dh, 128, 128, dtype=torch.float32, device=dev)
        ch = (2 * dg + dh) * 128
        tail = torch.zeros(n_seq, 3, ch, dtype=torch.bfloat16, device=dev)
        sbytes = t * (ch + 2 * dh * 128) * 2 + n_seq * (dh * 128 * 128 * 8 + 3 * ch * 4)
        cw, ab, nw = rnd(ch, 4), rnd(t, 2 * dh), torch.ones(128, dtype=torch.bfloat16, device=dev)
        gst, gtail = torch.zeros_like(st), torch.zeros_like(tail)
        a_log, dtb = torch.zeros(dh, device=dev), torch.zeros(dh, device=dev)
        if t <= 32:
            w_ab = rnd(2 * dh, width)
            like = lambda: gdn.decode_fused(dp[:, :ch + dh * 128], x16, w_ab, a_log, dtb, cw, gtail, gst, ar, nw, dh, dg)
        else:
            def like():
                mixed = basic.conv_silu(dp[:, :ch], cw, gtail[0])
                g, beta = basic.gdn_gates(ab, 0, dh, a_log, dtb, dh)
                o = gdn.chunked(mixed, 0, dg * 128, 2 * dg * 128, g, beta, gst[0], dh, dg)
                return basic.gated_rmsnorm(o.view(t * dh, 128), gate, nw)
            gate = rnd(t * dh, 128)
        pair("delta rule with convolution, decay, norm and gate", f"{t} tokens, {dh} heads x 128 x 128",
             (lambda: decay.delta_rule(dp, dw.m, st, tail, seg, pos1, dw.o.k), sbytes, 0), (like, sbytes, 0))
        del st, gst
        rst, gst = (torch.zeros(n_seq, rh, 128, 128, dtype=torch.float32, device=dev) for _ in range(2))
        rbytes = t * rh * 128 * 5 * 2 + n_seq * rh * 128 * 128 * 8
        mixed, gg, beta, gate2 = rnd(t, 3 * rh * 128), -torch.rand(t, rh, device=dev), torch.rand(t, rh, device=dev), rnd(t * rh, 128)
        core = (lambda: gdn.step(gst, ar, mixed, 0, rh * 128, 2 * rh * 128, gg, beta, rh, rh)) if t <= 32 else \
            (lambda: gdn.chunked(mixed, 0, rh * 128, 2 * rh * 128, gg, beta, gst[0], rh, rh))
        pair("retention with rotation, norm and gate (like: Gated DeltaNet, gated norm)", f"{t} tokens, {rh} heads x 128 x 128",
             (lambda: decay.retention(proj[:, pw.right_off:], pw.right, rst, seg, pos1, pw.right_o.k), rbytes, 0),
             (lambda: basic.gated_rmsnorm(core().view(t * rh, 128), gate2, nw), rbytes, 0))
        del rst, gst
        # ---- projections (like: none; all of them are the framework's GEMM)
        for what, pr in (("pair projection", pw.proj), ("delta projection", dw.proj), ("up projection", dense.up), ("down projection", dense.down),
                         ("side projection", dl.side_proj)):
            xk = rnd(t, pr.k)
            pair(what, f"{t} x {pr.n} x {pr.k}", (lambda: pr(xk), (pr.n * pr.k + t * pr.k + t * pr.n) * 2, 2 * t * pr.n * pr.k), None)
    # ---- prompt attention
    t = 8192
    table = (torch.arange(t // bs, dtype=torch.int32, device=dev) + 1)[None]
    q = rnd(t, H, 128)
    kc, vc = (rnd(t // bs + 1, bs, G * 128) for _ in range(2))
    k4, v4 = kc.view(-1, G, bs, 128), vc.view(-1, G, bs, 128)
    out = torch.empty(t, H * 128, dtype=torch.bfloat16, device=dev)
    pairs_n = sum(min(p + 1, window) for p in range(t))
    args = (i32([0]), i32([t]), i32([t]), t)
    pair("prompt attention (like: without bias)", f"{t} tokens, window {window}",
         (lambda: winattn.prefill(q, m, kc, vc, table, *args, out), 0, 2 * pairs_n * H * 256),
         (lambda: attention.prefill(q, k4, v4, table, *args, window=window), 0, 2 * pairs_n * H * 256))
    for b in (1, 32):
        tb = (torch.arange(b * pages, dtype=torch.int32, device=dev) + 1).view(b, pages)
        kc, vc = (rnd(b * pages + 1, bs, G * 128) for _ in range(2))
        k4, v4 = kc.view(-1, G, bs, 128), vc.view(-1, G, bs, 128)
        q, ob = rnd(b, H, 128), torch.empty(b, H * 128, dtype=torch.bfloat16, device=dev)
        pos, kvl, seen = i32([ctx - 1] * b), i32([ctx] * b), min(ctx, window)
        pair("decode attention (like: without bias)", f"batch {b}, window {seen}",
             (lambda: winattn.rows(q, m, kc, vc, tb, pos, ctx, ob), b * seen * G * 128 * 4, 0),
             (lambda: attention.decode(q, k4, v4, tb, kvl, max_kv_len=seen, window=window), b * seen * G * 128 * 4, 0))
    return rows_out


def run(args) -> dict:
    from ..ops import _lib
    from .clocks import ClockSampler
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    timer = _Timer(dev, args.steps, args.warmup)
    prompt, name = args.prompt, args.design
    out: dict = {"metric": f"{name} design: prefill and decode throughput", "unit": "tokens/s", "n_gpus": 1, "higher_is_better": True,
                 "steps": timer.steps, "warmup": timer.warmup, "dtype": "bf16", "data": "synthetic", "designs": {}}
    slots = 32
    sizes, models, kernels, closest = {
        "rutulix": (SIZES, _models, _kernels, "full-attention decoder, fp8 weights"),
        "zigasun": (ZG_SIZES, _zg_models, _zg_kernels, "Gated-DeltaNet / full-attention decoder, fp8 weights"),
        "kemirax": (KX_SIZES, _kx_models, _kx_kernels, "latent-attention decoder with routed experts, bf16 weights"),
        "nunosun": (NS_SIZES, _ns_models, _ns_kernels, "Gated-DeltaNet / full-attention decoder, fp8 weights")}[name]
    with torch.no_grad(), ClockSampler(0) as clk:
        for size in ([args.design_size] if args.design_size else list(sizes)):
            new, old = models(size, dev, prompt, slots)
            if name == "rutulix":
                width, heads, kv, dim, inter, chunk = SIZES[size]
                rec = {"layers": LAYERS, "width": width, "heads": heads, "kv_heads": kv, "dim": dim, "ff": inter * 3 // 2, "chunk": chunk}
            elif name == "zigasun":
                keys = ("width", "heads", "kv_heads", "dim", "vdim", "ff", "inner", "state", "dt_rank")
                rec = {"layers": LAYERS, **dict(zip(keys, ZG_SIZES[size]))}
            elif name == "nunosun":
                keys = ("width", "heads", "kv_heads", "window", "retention_heads", "delta_heads", "delta_kv_heads", "swiglu_ff", "experts", "top", "side")
                rec = {"layers": NS_LAYERS, **dict(zip(keys, NS_SIZES[size]))}
            else:
                keys = ("width", "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "gla_heads", "ff", "experts", "identity", "top")
                rec = {"layers": KX_LAYERS, **dict(zip(keys, KX_SIZES[size]))}
            rec.update({"prompt": prompt, name: _throughput(new, dev, prompt, slots, timer)})
            torch.cuda.empty_cache()
            rec[f"closest ({closest})"] = _throughput(old, dev, prompt, slots, timer)
            torch.cuda.empty_cache()
            rec["kernels"] = kernels(size, dev, timer, prompt)
            torch.cuda.empty_cache()
            out["designs"][size] = rec
            _lib.check_status()
    first = next(iter(out["designs"].values()))
    out["value"] = first[name]["prefill_tok_s"]
    out["clocks"] = clk.summary()
    out["config"] = {"l2": "flushed before every timed call", "roofline": _peaks()[1], "prompt": prompt, "decode_batch": slots}
    return out
