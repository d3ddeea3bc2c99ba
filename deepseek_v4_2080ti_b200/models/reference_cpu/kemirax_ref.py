"""Plain statement of the Kemirax decoder in PyTorch, one function per mechanism, whole sequences at once.

Nothing here is shared with the serving path (``models/kemirax.py``, ``ops/``): the tests compare the two.  Every
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


def log_sigmoid(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, max=0) - torch.log1p(torch.exp(-x.abs()))


def token_shift(h: torch.Tensor, amount: torch.Tensor) -> torch.Tensor:
    """h [T, C]: every row moves towards the row before it (zeros before the first) by ``amount`` per channel."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * amount


# ---------------------------------------------------------------------------------------------- latent attention
def yarn_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """(fp64 frequencies, factor on cosine and sine) of a rotation {dims, base, scaling or nothing}."""
    d, base, s = rot["dims"], rot["base"], rot.get("scaling")
    out = []
    for i in range(d // 2):
        f = base ** (-2.0 * i / d)
        if s:
            at = [d * math.log(s["original"] / (2 * math.pi * s[n])) / (2 * math.log(base)) for n in ("fast", "slow")]
            lo, hi = max(math.floor(at[0]), 0), min(math.ceil(at[1]), d - 1)
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / s["factor"] * r + f * (1.0 - r)
        out.append(f)
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0 if s else 1.0


def rotate_half(x: torch.Tensor, positions, rot: dict) -> torch.Tensor:
    """x [T, ..., R]: the first rot["dims"] values of the last dimension in pairs (i, i + dims / 2)."""
    f, m = yarn_frequencies(rot)
    half = rot["dims"] // 2
    a = torch.as_tensor(positions, dtype=torch.float64)[:, None] * f[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    c, s = (m * torch.cos(a)).to(x.dtype).view(shape), (m * torch.sin(a)).to(x.dtype).view(shape)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def causal_softmax(scores: torch.Tensor) -> torch.Tensor:
    """scores [T, T] -> weights; row i sees columns up to i."""
    n = scores.shape[0]
    hidden = torch.arange(n)[None, :] > torch.arange(n)[:, None]
    s = scores.masked_fill(hidden, float("-inf"))
    p = torch.exp(s - s.max(-1, keepdim=True).values)
    return p / p.sum(-1, keepdim=True)


def latent_keys(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """What a layer caches: (normalised latent [T, kv_rank], rotated key part [T, rot_dim])."""
    z = h @ w["dkv"].t()
    r = mix["kv_rank"]
    return rms(z[:, :r], eps) * w["dkv.norm"], rotate_half(z[:, r:], range(h.shape[0]), mix["rot"])


def latent_attention(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float, c: torch.Tensor, kr: torch.Tensor) -> torch.Tensor:
    """h [T, width] -> [T, width]; c, kr of this layer or of the one it borrows from."""
    n, heads, d, r, v = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    q = ((rms(h @ w["dq"].t(), eps) * w["dq.norm"]) @ w["uq"].t()).view(n, heads, d + r)
    qr = rotate_half(q[:, :, d:], range(n), mix["rot"])
    keys, values = (c @ w["uk"].t()).view(n, heads, d), (c @ w["uv"].t()).view(n, heads, v)
    out = []
    for i in range(heads):
        s = (q[:, i, :d] @ keys[:, i].t() + qr[:, i] @ kr.t()) * mix["scale"]
        out.append(causal_softmax(s) @ values[:, i])
    return torch.cat(out, -1) @ w["o"].t()


# ---------------------------------------------------------------------------------------------- gated linear attention
def gated_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, log_decay: torch.Tensor,
                     state: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """q, k, log_decay [T, H, D], v [T, H, V], one token after the other:  S <- exp(log_decay) S + k v^T (the decay per row
    of S), o = S^T q.  Returns (o [T, H, V], final state [H, D, V])."""
    s = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]) if state is None else state.clone()
    rows = []
    for t in range(q.shape[0]):
        s = torch.exp(log_decay[t])[:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hdv,hd->hv", s, q[t]))
    return torch.stack(rows), s


def linear_attention(h: torch.Tensor, w: dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    """h [T, width] -> [T, width]."""
    n, heads, d, vd = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = (h @ w["q"].t()).view(n, heads, d) * d ** -0.5
    k = (h @ w["k"].t()).view(n, heads, d)
    v = (h @ w["v"].t()).view(n, heads, vd)
    z = (h @ w["a1"].t()) @ w["a2"].t() + w["a2.b"]
    o, _ = gated_recurrence(q, k, v, (log_sigmoid(z) / mix["tau"]).view(n, heads, d))
    o = (rms(o, eps) * w["norm"]).reshape(n, -1)
    g = h @ w["g"].t()
    return (o * g * sigmoid(g)) @ w["o"].t()


# ---------------------------------------------------------------------------------------------- feed-forward
def clamped_unit(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ gate.t(), max=limit)
    u = torch.clamp(h @ up.t(), -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.t()


def choose(logits: torch.Tensor, correction: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """logits [T, E] -> (chosen experts [T, top], their softmax scores): the correction takes part in the choice only."""
    e = torch.exp(logits - logits.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    idx = torch.topk(s + correction, top, dim=-1).indices
    return idx, torch.gather(s, 1, idx)


def experts(h: torch.Tensor, w: dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    """Routed experts, identity experts and the gated shared expert."""
    r = mlp["router"]
    idx, wt = choose(h @ w["router"].t(), w["correction"], r["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(r["top"]):
            e = int(idx[t, j])
            if e < r["experts"]:
                y = clamped_unit(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], mlp["expert"]["limit"])[0]
            else:
                y = h[t]
            out[t] += wt[t, j] * y
    if mlp.get("shared"):
        y = clamped_unit(h, w["shared.gate"], w["shared.up"], w["shared.down"], mlp["shared"]["limit"])
        out = out + sigmoid(h @ w["shared.sg"].t()) * y
    return out


# ---------------------------------------------------------------------------------------------- the decoder
def forward(cfg: dict, tensors: dict[str, torch.Tensor], tokens, dtype=torch.float64, taps: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence.  ``taps`` receives the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]

    def sub(prefix):
        return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    cached = {}
    for i, L in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", L["mixer"]
        h = rms(x, eps) * w[p + "norm1"]
        m = token_shift(h, w[p + "shift"])
        t = sub(p + "mix.")
        if L["type"] == "latent_attention":
            src = mix.get("kv_from")
            if src is None:
                cached[i] = latent_keys(m, t, mix, eps)
            y = latent_attention(m, t, mix, eps, *cached[i if src is None else src])
        else:
            y = linear_attention(m, t, mix, eps)
        x = x + y * sigmoid(h @ w[p + "rg1"].t() + w[p + "rg1.b"])
        if L.get("mlp"):
            x = x + experts(h, sub(p + "mlp."), L["mlp"]) * sigmoid(h @ w[p + "rg2"].t() + w[p + "rg2.b"])
        if taps is not None:
            taps.append(x.clone())
    return rms(x, eps) * w["final.norm"] @ w["head"].t()
