"""Plain statement of the Nunosun decoder in PyTorch, one function per mechanism, whole sequences at once.

Nothing here is shared with the serving path (``models/nunosun.py``, ``ops/``): the tests compare the two.  Every
function takes and returns ordinary tensors in the dtype it is given (the tests use fp64 and fp32).
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [T, C], w [C, taps] (last column: the row itself) -> [T, C]; rows before the first are zero."""
    taps = w.shape[1]
    full = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(full[j:j + x.shape[0]] * w[:, j] for j in range(taps))


# ---------------------------------------------------------------------------------------------- windowed attention
def bucket(n: int, rows: int, reach: int) -> int:
    """Row of the bias table for a key n positions back: one row per distance in the lower half, logarithmic up to ``reach``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def window_attention(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    """h [T, width] -> [T, width]."""
    n, heads, groups, d, v = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms((h @ w["q"].t()).view(n, heads, d), eps) * w["q.norm"]
    k = rms((h @ w["k"].t()).view(n, groups, d), eps) * w["k.norm"]
    val = (h @ w["v"].t()).view(n, groups, v)
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    hidden = (back < 0) | (back >= mix["mask"]["size"])
    table = torch.tensor([bucket(i, w["rel"].shape[0], mix["bias_max"]) for i in range(n)])
    bias = w["rel"][table[back.clamp(min=0)]]                                     # [T, T, heads]
    out = []
    for i in range(heads):
        g = i // (heads // groups)
        s = ((q[:, i] @ k[:, g].t()) * mix["scale"] + bias[:, :, i]).masked_fill(hidden, float("-inf"))
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append(p / p.sum(-1, keepdim=True) @ val[:, g])
    return torch.cat(out, -1) @ w["o"].t()


# ---------------------------------------------------------------------------------------------- retention
def rotate_half(x: torch.Tensor, positions, dims: int, base: float) -> torch.Tensor:
    """x [T, ..., D]: the first ``dims`` values of the last dimension in pairs (i, i + dims / 2)."""
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = torch.as_tensor(positions, dtype=torch.float64)[:, None] * f[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    c, s = torch.cos(a).to(x.dtype).view(shape), torch.sin(a).to(x.dtype).view(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def retention_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor,
                         state: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """q, k [T, H, D], v [T, H, V], decay [H]:  S <- decay S + k v^T,  o = S^T q.  Returns (o [T, H, V], S [H, D, V])."""
    s = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]) if state is None else state.clone()
    rows = []
    for t in range(q.shape[0]):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hdv,hd->hv", s, q[t]))
    return torch.stack(rows), s


def retention(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    """h [T, width] -> [T, width]."""
    n, heads, d, v = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    rot = lambda z: rotate_half(z.view(n, heads, d), range(n), mix["rot"]["dims"], mix["rot"]["base"])
    q, k = rot(h @ w["q"].t()), rot(h @ w["k"].t()) * d ** -0.5
    o, _ = retention_recurrence(q, k, (h @ w["v"].t()).view(n, heads, v), torch.tensor(mix["decay"], dtype=torch.float64).to(h.dtype))
    return (rms(o, eps).reshape(n, -1) * silu(h @ w["g"].t())) @ w["o"].t()


def side_by_side(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    """Windowed attention and retention on the same rows; the mean of the two, each normalised over the width."""
    sub = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}
    left = rms(window_attention(h, sub("left."), mix["left"], eps), eps) * w["left.out"]
    right = rms(retention(h, sub("right."), mix["right"], eps), eps) * w["right.out"]
    return 0.5 * (left + right)


# ---------------------------------------------------------------------------------------------- gated delta rule
def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, log_decay: torch.Tensor, beta: torch.Tensor,
                     state: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """q, k [T, H, D], v [T, H, V], log_decay, beta [T, H], one token after the other: S <- exp(log_decay) S,
    S <- S + k (beta (v - S^T k))^T, o = S^T q.  Returns (o [T, H, V], S [H, D, V])."""
    s = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]) if state is None else state.clone()
    rows = []
    for t in range(q.shape[0]):
        s = torch.exp(log_decay[t])[:, None, None] * s
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        rows.append(torch.einsum("hdv,hd->hv", s, q[t]))
    return torch.stack(rows), s


def delta_mixer(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    """h [T, width] -> [T, width]."""
    n, heads, groups, d, v = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q, k, val = (silu(causal_conv(h @ w[x].t(), w[x + ".conv"])) for x in ("q", "k", "v"))
    spread = lambda x: unit(x.view(n, groups, d)).repeat_interleave(heads // groups, 1)
    log_decay = -torch.exp(w["A_log"]) * softplus(h @ w["a"].t() + w["dt_bias"])
    o, _ = delta_recurrence(spread(q) * d ** -0.5, spread(k), val.view(n, heads, v), log_decay, sigmoid(h @ w["b"].t()))
    return ((rms(o, eps) * w["norm"]).reshape(n, -1) * silu(h @ w["g"].t())) @ w["o"].t()


# ---------------------------------------------------------------------------------------------- feed-forward
def poly_norm(z: torch.Tensor, c: torch.Tensor, eps: float) -> torch.Tensor:
    """c[0] N(z) + c[1] N(z^2) + c[2] N(z^3) + c[3], N: over the root mean square of the row."""
    return c[0] * rms(z, eps) + c[1] * rms(z * z, eps) + c[2] * rms(z * z * z, eps) + c[3]


def dense(h: torch.Tensor, w: dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    return poly_norm(h @ w["up"].t(), w["act"], eps) @ w["down"].t()


def choose(logits: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """logits [T, E] -> (the ``top`` largest [T, top], softmax over them)."""
    z, idx = torch.topk(logits, top, dim=-1)
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    return idx, e / e.sum(-1, keepdim=True)


def experts(h: torch.Tensor, w: dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    idx, wt = choose(h @ w["router"].t() + w["router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, j = torch.nonzero(idx == e, as_tuple=True)
        if t.numel():
            x = h[t]
            y = (silu(x @ w[f"e{e}.gate"].t()) * (x @ w[f"e{e}.up"].t())) @ w[f"e{e}.down"].t()
            out.index_add_(0, t, wt[t, j][:, None] * y)
    return out


# ---------------------------------------------------------------------------------------------- token input of a layer
def token_input(x: torch.Tensor, e: torch.Tensor, w: dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    """What a layer adds to the residual x [T, width] for its part e [T, dim] of the tokens' side embedding."""
    return rms((gelu_tanh(x @ w["gate"].t()) * e) @ w["proj"].t(), eps) * w["norm"]


# ---------------------------------------------------------------------------------------------- the decoder
def forward(cfg: dict, tensors: dict[str, torch.Tensor], tokens, dtype=torch.float64, taps: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence.  ``taps`` receives the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps, dim = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    sub = lambda prefix: {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = rms(w["embed"][ids], eps) * w["embed.norm"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        m = h + causal_conv(h, w[p + "canon1"])
        y = (delta_mixer if L["type"] == "delta" else side_by_side)(m, sub(p + "mix."), L["mixer"], eps)
        if L.get("mlp"):
            f = sub(p + "mlp.")
            y = y + (experts(h, f, L["mlp"]) if L["mlp"]["kind"] == "moe" else dense(h, f, eps))
        x = x + y
        x = x + token_input(x, w["side.embed"][ids, i * dim:(i + 1) * dim], sub(p + "side."), eps)
        if taps is not None:
            taps.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].t() * cfg["logit_scale"]
