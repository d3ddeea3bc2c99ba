"""Plain statement of the Zigasun decoder in PyTorch, one function per mechanism, whole sequences at once.

Nothing here is shared with the serving path (``models/zigasun.py``, ``ops/``): the tests compare the two.  Every
function takes and returns ordinary tensors in the dtype it is given (the tests use fp64 and fp32).
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, K] (the last column multiplies the current row), zeros before the first row."""
    k = taps.shape[1]
    out = torch.zeros_like(x) + bias
    for j in range(k):
        back = k - 1 - j
        if back < x.shape[0]:
            out[back:] = out[back:] + x[:x.shape[0] - back] * taps[:, j]
    return out


def silu(x: torch.Tensor) -> torch.Tensor:
    return x / (1.0 + torch.exp(-x))


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def selective_scan(x: torch.Tensor, dt: torch.Tensor, a: torch.Tensor, b: torch.Tensor, c: torch.Tensor, d: torch.Tensor,
                   state: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """x, dt [T, C]; a [C, N] (negative); b, c [T, N]; d [C].  Per channel and state, one token after the other:
    S <- exp(dt a) S + dt x b, y = sum over the states of S c, plus d x.  Returns (y [T, C], final state [C, N])."""
    s = torch.zeros_like(a) if state is None else state.clone()
    rows = []
    for t in range(x.shape[0]):
        s = torch.exp(dt[t][:, None] * a) * s + (dt[t] * x[t])[:, None] * b[t][None, :]
        rows.append((s * c[t][None, :]).sum(-1) + d * x[t])
    return torch.stack(rows), s


def scan_mixer(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict) -> torch.Tensor:
    """h [T, width] -> [T, width].  ``w``: the mixer's tensors by short name."""
    inner, rank, n = mix["inner"], mix["dt_rank"], mix["state"]
    xz = h @ w["in"].t()
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w["conv"], w["conv.b"]))
    p = x @ w["x"].t()
    dt = softplus(p[:, :rank] @ w["dt"].t() + w["dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(w["A_log"]), p[:, rank:rank + n], p[:, rank + n:], w["D"])
    return (y * silu(z)) @ w["o"].t()


def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    """fp64 factor per position: grows with the logarithm of the number of whole ``every`` blocks passed."""
    return torch.tensor([1.0 + coef * math.log(math.floor((int(p) + 1) / every) + 1.0) for p in positions], dtype=torch.float64)


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """One causal map: q, k [T, d], v [T, dv] -> [T, dv]."""
    s = q @ k.t() * scale
    n = q.shape[0]
    hidden = torch.arange(n)[None, :] > torch.arange(n)[:, None]
    s = s.masked_fill(hidden, float("-inf"))
    p = torch.exp(s - s.max(-1, keepdim=True).values)
    return p / p.sum(-1, keepdim=True) @ v


def lambda_of(w: dict[str, torch.Tensor], diff: float) -> torch.Tensor:
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def difference_of_maps(a1: torch.Tensor, a2: torch.Tensor, lam: torch.Tensor, diff: float, eps: float) -> torch.Tensor:
    """a1, a2 [..., dv]: the second map is subtracted, the difference normalised over dv and scaled."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def keys_values(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """(k [T, G, 2, dim] normalised per head and map, v [T, G, vdim])."""
    n, g = h.shape[0], mix["kv_heads"]
    k = rms((h @ w["k"].t()).view(n, g, 2, mix["dim"]), eps) * w["k.norm"]
    return k, (h @ w["v"].t()).view(n, g, mix["vdim"])


def attention_mixer(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float, k: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
    """h [T, width] -> [T, width]; k, v of this layer or of the one it borrows from."""
    n, heads = h.shape[0], mix["heads"]
    per = heads // mix["kv_heads"]
    q = rms((h @ w["q"].t()).view(n, heads, 2, mix["dim"]), eps) * w["q.norm"]
    if mix.get("q_temp"):
        f = query_temperature(torch.arange(n), mix["q_temp"]["coef"], mix["q_temp"]["every"])
        q = q * f.to(q.dtype)[:, None, None, None]
    lam = lambda_of(w, mix["diff"])
    out = []
    for i in range(heads):
        a1, a2 = (softmax_attention(q[:, i, m], k[:, i // per, m], v[:, i // per], mix["scale"]) for m in (0, 1))
        out.append(difference_of_maps(a1, a2, lam, mix["diff"], eps))
    gate = 1.0 / (1.0 + torch.exp(-(h @ w["g"].t())))                 # [T, heads]
    o = torch.stack(out, 1) * gate[:, :, None]
    return o.reshape(n, -1) @ w["o"].t()


def clamped_glu(h: torch.Tensor, w: dict[str, torch.Tensor], limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w["gate"].t(), max=limit)
    u = torch.clamp(h @ w["up"].t(), -limit, limit)
    return (g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)) @ w["down"].t()


def forward(cfg: dict, tensors: dict[str, torch.Tensor], tokens, dtype=torch.float64, taps: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence.  ``taps`` receives the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    cache = {}
    for i, L in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", L["mixer"]
        if L["type"] == "attention":
            if mix.get("kv_from") is None:
                cache[i] = keys_values(x, sub(p + "mix."), mix, eps)
            k, v = cache[i if mix.get("kv_from") is None else mix["kv_from"]]
            y = attention_mixer(x, sub(p + "mix."), mix, eps, k, v)
        else:
            y = scan_mixer(x, sub(p + "mix."), mix)
        x = x + m * rms(y, eps) * w[p + "norm1"]
        if L.get("mlp"):
            x = x + m * rms(clamped_glu(x, sub(p + "mlp."), L["mlp"]["limit"]), eps) * w[p + "norm2"]
        if taps is not None:
            taps.append(x.clone())
    return rms(x, eps) * w["final.norm"] @ w["head"].t()
