"""A plain, slow implementation of the Kikopel decoder, one function per mechanism.

Written from the design's equations in torch on the CPU (float64 by default), it shares
no code with the package: it takes the ``config.json`` dictionary and a dictionary of
tensors by checkpoint name, and runs one whole sequence at once (the recurrence token by
token).

Notation: n tokens, width D, positions p from 0; latent attention: H heads, d unrotated and
dr rotated query / key numbers, values of e numbers, a latent of r numbers; recurrence:
Hr heads with dk key channels and dv value numbers and a forget factor per key channel.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """rms(x) times a vector, or times one number for all coordinates."""
    return rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def pair_rows(tokens: torch.Tensor, buckets: int, mul_prev: int, mul_cur: int) -> torch.Tensor:
    """The pair table's row of every token: (before * mul_prev + own * mul_cur) mod buckets, and row ``buckets`` for the first."""
    rows = [buckets]
    ids = tokens.tolist()
    for before, own in zip(ids[:-1], ids[1:]):
        rows.append((before * mul_prev + own * mul_cur) % buckets)
    return torch.tensor(rows)


def embed(tokens: torch.Tensor, table, scale: float, pairs=None, pair_cfg: Optional[dict] = None) -> torch.Tensor:
    """Rows of the table times ``scale`` plus rows of the pair table as they are."""
    x = table[tokens] * scale
    if pairs is not None:
        x = x + pairs[pair_rows(tokens, pair_cfg["buckets"], pair_cfg["mul_prev"], pair_cfg["mul_cur"])]
    return x


def turn(x: torch.Tensor, base: float, first: int = 0) -> torch.Tensor:
    """x [n, ..., dr]: entries i and i + dr/2 of position p turn by p base^(-2i/dr)."""
    dr = x.shape[-1]
    out = x.clone()
    p = torch.arange(first, first + x.shape[0], dtype=x.dtype)
    for i in range(dr // 2):
        a = p * base ** (-2.0 * i / dr)
        c, s = torch.cos(a), torch.sin(a)
        while c.dim() < x.dim() - 1:
            c, s = c[:, None], s[:, None]
        u, v = x[..., i], x[..., i + dr // 2]
        out[..., i] = u * c - v * s
        out[..., i + dr // 2] = v * c + u * s
    return out


def visible(n: int, window: Optional[int]) -> torch.Tensor:
    """[n, n] bool: query i sees key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    vis = j <= i
    return vis if window is None else vis & (i - j < window)


def softmax_over(scores: torch.Tensor, vis: torch.Tensor) -> torch.Tensor:
    return torch.softmax(scores.masked_fill(~vis[None], -float("inf")), dim=-1)


def latent_attention(h, t: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    H, d, dr, e, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    cq = norm(h @ t[pre + "dq"].T, t[pre + "dq.norm"], eps)
    q = (cq @ t[pre + "uq"].T).reshape(n, H, d + dr)
    qa, qr = q[..., :d], turn(q[..., d:], base)
    down = h @ t[pre + "dkv"].T
    c = norm(down[:, :r], t[pre + "dkv.norm"], eps)
    kr = turn(down[:, r:], base)
    k = (c @ t[pre + "uk"].T).reshape(n, H, d)
    v = (c @ t[pre + "uv"].T).reshape(n, H, e)
    scores = (torch.einsum("ihd,jhd->hij", qa, k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    w = softmax_over(scores, visible(n, (m.get("mask") or {}).get("size")))
    y = torch.einsum("hij,jhe->ihe", w, v).reshape(n, H * e)
    return (y * torch.sigmoid(h @ t[pre + "g"].T)) @ t[pre + "o"].T


def forget_factors(h, t, pre: str, m: dict) -> torch.Tensor:
    """[n, Hr, dk]: l + (1 - l) sigmoid(W h + b), between the channel's lower bound l and one."""
    low = t[pre + "lower"]
    f = low + (1 - low) * torch.sigmoid(h @ t[pre + "f"].T + t[pre + "f.b"])
    return f.reshape(h.shape[0], m["heads"], m["dim"])


def forgetting_outer_products(q, v, f, state: Optional[torch.Tensor] = None):
    """q, f [n, Hr, dk], v [n, Hr, dv]; token by token S <- f_t (rows) * S + (1 - f_t) v_t^T and o_t = S^T q_t.
    Returns (o [n, Hr, dv], the last S [Hr, dk, dv])."""
    n, Hr, dk = q.shape
    S = torch.zeros((Hr, dk, v.shape[2]), dtype=q.dtype) if state is None else state.clone()
    out = []
    for i in range(n):
        S = f[i][:, :, None] * S + (1 - f[i])[:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[i]))
    return torch.stack(out), S


def hgrn2(h, t, pre: str, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    Hr, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ t[pre + "q"].T).reshape(n, Hr, dk)
    v = (h @ t[pre + "v"].T).reshape(n, Hr, dv)
    o, _ = forgetting_outer_products(q, v, forget_factors(h, t, pre, m))
    return norm(o, t[pre + "norm"], eps).reshape(n, Hr * dv) @ t[pre + "o"].T


def poly_norm(z: torch.Tensor, coefficients: torch.Tensor, eps: float) -> torch.Tensor:
    """a rms(z) + b rms(z^2) + c rms(z^3) + e, powers element by element."""
    a, b, c, e = coefficients
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def feed_forward(h, t, pre: str, eps: float) -> torch.Tensor:
    return poly_norm(h @ t[pre + "up"].T, t[pre + "act"], eps) @ t[pre + "down"].T


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens, dtype=torch.float64, taps: Optional[List[torch.Tensor]] = None
            ) -> torch.Tensor:
    """Logits [n, vocab]; ``taps`` receives the stream after every layer."""
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps, mult = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    emb = cfg.get("embedding") or {}
    toks = torch.as_tensor(list(tokens), dtype=torch.long)
    x = embed(toks, t["embed"], emb.get("scale", 1.0), t.get("bigram") if emb.get("bigram") else None, emb.get("bigram"))
    for i, L in enumerate(cfg["layers"]):
        pre = f"l{i}."
        mixer = {"latent_attention": latent_attention, "hgrn2": hgrn2}[L["type"]]
        x = x + mult * norm(mixer(x, t, pre + "mix.", L["mixer"], eps), t[pre + "norm1"], eps)
        if L.get("mlp") is not None:
            x = x + mult * norm(feed_forward(x, t, pre + "mlp.", eps), t[pre + "norm2"], eps)
        if taps is not None:
            taps.append(x.clone())
    return norm(x, t["final.norm"], eps) @ t["head"].T
