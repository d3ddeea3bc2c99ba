"""Plain statement of the Rutulix decoder in PyTorch, one function per mechanism, whole sequences at once.

Nothing here is shared with the serving path (``models/rutulix.py``, ``ops/``): the tests compare the two.  Every
function takes and returns ordinary tensors in the dtype it is given (the tests use fp64 and fp32).
"""
from __future__ import annotations

import math

import torch


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """Centred norm with a weight and no bias; the variance is the mean of the squared deviations."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def yarn_frequencies(dims: int, base: float, scaling: dict | None) -> tuple[list[float], float]:
    """(frequency of each rotated pair, factor on cos and sin)."""
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freqs, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def dim_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(dim_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_interleaved(x: torch.Tensor, positions: torch.Tensor, freqs: list[float], mscale: float) -> torch.Tensor:
    """x [T, heads, dim]: the pair (2i, 2i + 1) of every head turns by position * freqs[i]; dims past the pairs stay."""
    out = x.clone()
    for i, f in enumerate(freqs):
        a = (positions.double() * f)[:, None]
        c, s = (a.cos() * mscale).to(x.dtype), (a.sin() * mscale).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def chunk_visible(n: int, size: int | None) -> torch.Tensor:
    """[n, n] bool: may position i (row) look at position j (column)?  Causal, and only inside i's chunk of ``size``
    positions (counted from the start of the sequence)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    ok = j <= i
    if size:
        ok = ok & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))
    return ok


def talking_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, talk: torch.Tensor, scale: float,
                      visible: torch.Tensor) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv].  The scaled scores of the H heads are mixed by ``talk``
    [H, H] before the mask and the softmax."""
    heads, groups = q.shape[1], k.shape[1]
    kv_of = [h // (heads // groups) for h in range(heads)]
    raw = torch.stack([q[:, h] @ k[:, kv_of[h]].t() * scale for h in range(heads)])        # [H, T, T]
    mixed = torch.einsum("hg,gij->hij", talk, raw)
    p = mixed.masked_fill(~visible[None], float("-inf")).softmax(-1)
    return torch.stack([p[h] @ v[:, kv_of[h]] for h in range(heads)], 1)


def attention_mixer(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    """h [T, width] (the normalised input of the mixer) -> [T, width].  ``w``: the mixer's tensors by short name."""
    n = h.shape[0]
    heads, groups, dim = mix["heads"], mix["kv_heads"], mix["dim"]
    q, k = h @ w["q"].t(), h @ w["k"].t()
    v = k.view(n, groups, dim)                                   # the raw key projection is the value
    q = rms_norm(q, w["q.norm"], eps).view(n, heads, dim)
    k = rms_norm(k, w["k.norm"], eps).view(n, groups, dim)
    rot = mix.get("rot")
    if rot:
        freqs, ms = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        pos = torch.arange(n)
        q, k = rotate_interleaved(q, pos, freqs, ms), rotate_interleaved(k, pos, freqs, ms)
    size = (mix.get("mask") or {}).get("size")
    o = talking_attention(q, k, v, w["talk"], mix["scale"], chunk_visible(n, size))
    return o.reshape(n, -1) @ w["o"].t()


def xielu(z: torch.Tensor, act: torch.Tensor) -> torch.Tensor:
    """Two-branch activation with parameters (p, q): quadratic for positive inputs, exponential otherwise."""
    ap, an = torch.nn.functional.softplus(act[0]), 0.5 + torch.nn.functional.softplus(act[1])
    zn = z.clamp(max=0.0)
    return torch.where(z > 0, ap * z * z + 0.5 * z, an * (torch.expm1(zn) - zn) + 0.5 * z)


def dense_mlp(h: torch.Tensor, w: dict[str, torch.Tensor]) -> torch.Tensor:
    return xielu(h @ w["up"].t() + w["up.b"], w["act"]) @ w["down"].t() + w["down.b"]


def layer_runs(n_layers: int, loop: dict | None) -> list[tuple[int, int | None]]:
    """Order of execution: (layer, number of the pass that begins right before it or None)."""
    if not loop:
        return [(i, None) for i in range(n_layers)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out: list[tuple[int, int | None]] = [(i, None) for i in range(a)]
    for t in range(times):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n_layers)]


def forward(cfg: dict, tensors: dict[str, torch.Tensor], tokens, dtype=torch.float64, taps: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence.  ``taps`` receives the residual stream after every layer run."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, begins in layer_runs(len(cfg["layers"]), cfg.get("loop")):
        if begins is not None:
            x = x + w["loop.step"][begins]
        L, p = cfg["layers"][i], f"l{i}."
        y = attention_mixer(layer_norm(x, w[p + "norm1"], eps), sub(p + "mix."), L["mixer"], eps)
        x = x + layer_norm(y, w[p + "norm1b"], eps)
        if L.get("mlp"):
            y = dense_mlp(layer_norm(x, w[p + "norm2"], eps), sub(p + "mlp."))
            x = x + layer_norm(y, w[p + "norm2b"], eps)
        if taps is not None:
            taps.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].t()
