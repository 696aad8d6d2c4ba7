"""A plain, slow implementation of the Saposun decoder, one function per mechanism.

Written from the design's equations in torch on the CPU (float64 by default), it shares
no code with the package: it takes the ``config.json`` dictionary and a dictionary of
tensors by checkpoint name, and runs one whole sequence at once (the recurrence token by
token).

Notation: n tokens, width D, positions p from 0; latent attention: H heads of d unrotated
and dr rotated query / key numbers, values of e numbers, a latent of r numbers; softmax
attention: H query heads, G key/value heads, head size d (queries, keys) and e (values);
retention: Hr heads with keys of dk and values of dv numbers.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def turn(x: torch.Tensor, base: float, dims: int, halves: bool, first: int = 0) -> torch.Tensor:
    """x [n, heads, size] at the positions first, first + 1, ...: pair i of the first ``dims`` elements of every head turns
    by p base^(-2i/dims); a pair is the elements (i, i + dims/2) for ``halves``, else (2i, 2i + 1)."""
    out = x.clone()
    p = torch.arange(first, first + x.shape[0], dtype=x.dtype)
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if halves else (2 * i, 2 * i + 1)
        ang = (p * base ** (-2.0 * i / dims))[:, None]
        u, v = x[:, :, a], x[:, :, b]
        out[:, :, a] = u * torch.cos(ang) - v * torch.sin(ang)
        out[:, :, b] = v * torch.cos(ang) + u * torch.sin(ang)
    return out


def in_window(n: int, size: Optional[int]) -> torch.Tensor:
    """[n, n] booleans: row i sees column j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) if size is None else (j <= i) & (i - j < size)


def softmax_over(scores: torch.Tensor, vis: torch.Tensor) -> torch.Tensor:
    """scores [H, n, m], vis [n, m]: an ordinary softmax over the visible columns."""
    return torch.softmax(scores.masked_fill(~vis[None], -math.inf), -1)


# ---- latent attention ---------------------------------------------------------------------------------------------------
def latent_rows(h, t: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """What is cached: the latents [n, r] and the key part that all heads share [n, dr], turned."""
    r = m["kv_rank"]
    z = h @ t[pre + "dkv"].T
    return norm(z[:, :r], t[pre + "dkv.norm"], eps), turn(z[:, None, r:], m["rot"]["base"], m["rot"]["dims"], False)[:, 0]


def latent_attention(h, t, pre: str, m: dict, eps: float, rows: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    """``rows``: :func:`latent_rows` of this layer or of the layer whose rows it reads."""
    n = h.shape[0]
    H, d, dr, e = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = rows
    q = (norm(h @ t[pre + "dq"].T, t[pre + "dq.norm"], eps) @ t[pre + "uq"].T).reshape(n, H, d + dr)
    qr = turn(q[:, :, d:], m["rot"]["base"], m["rot"]["dims"], False)
    k = (c @ t[pre + "uk"].T).reshape(n, H, d)
    v = (c @ t[pre + "uv"].T).reshape(n, H, e)
    s = (torch.einsum("ihd,jhd->hij", q[:, :, :d], k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    w = softmax_over(s, in_window(n, m["mask"]["size"] if m.get("mask") else None))
    return torch.einsum("hij,jhe->ihe", w, v).reshape(n, H * e) @ t[pre + "o"].T


# ---- retention ----------------------------------------------------------------------------------------------------------
def decaying_outer_products(q, k, v, decay, state: Optional[torch.Tensor] = None):
    """q, k [n, Hr, dk], v [n, Hr, dv], decay [Hr]; token by token S <- decay S + k_t v_t^T and o_t = S^T q_t.
    Returns (o [n, Hr, dv], the last S [Hr, dk, dv])."""
    n, Hr, dk = q.shape
    S = torch.zeros((Hr, dk, v.shape[2]), dtype=q.dtype) if state is None else state.clone()
    out = []
    for i in range(n):
        S = decay[:, None, None] * S + k[i][:, :, None] * v[i][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[i]))
    return torch.stack(out), S


def retention(h, t, pre: str, m: dict, eps: float) -> torch.Tensor:
    n = h.shape[0]
    Hr, dk, dv = m["heads"], m["dim"], m["vdim"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = turn((h @ t[pre + "q"].T).reshape(n, Hr, dk), base, dims, True)
    k = turn((h @ t[pre + "k"].T).reshape(n, Hr, dk), base, dims, True) * dk ** -0.5
    v = (h @ t[pre + "v"].T).reshape(n, Hr, dv)
    o, _ = decaying_outer_products(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o, eps).reshape(n, Hr * dv) * silu(h @ t[pre + "g"].T)) @ t[pre + "o"].T


# ---- attention with a window and pooled blocks ------------------------------------------------------------------------------
def causal_filter(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [n, channels], w [channels, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    n, taps = u.shape[0], w.shape[1]
    z = torch.cat([torch.zeros((taps - 1, u.shape[1]), dtype=u.dtype), u])
    return sum(w[:, j] * z[j:j + n] for j in range(taps))


def pooled(x: torch.Tensor, P: int) -> torch.Tensor:
    """x [n, heads, size] -> the means of whole blocks of P positions [n // P, heads, size]."""
    b = x.shape[0] // P
    return x[:b * P].reshape(b, P, *x.shape[1:]).mean(1)


def sees_block(n: int, size: int, P: int) -> torch.Tensor:
    """[n, n // P]: block b (positions bP .. bP + P - 1) lies wholly before the window of row i."""
    i, b = torch.arange(n)[:, None], torch.arange(n // P)[None, :]
    return b * P + P - 1 <= i - size


def capped(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap else s


def projected(h, t, pre: str, m: dict, eps: float):
    """(q [n, H, d], k [n, G, d], v [n, G, e]): projections, short filters, rotation, the values' norm."""
    n = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def make(name, heads, size):
        u = h @ t[pre + name].T
        if m.get("conv"):
            u = causal_filter(u, t[pre + name + ".conv"])
        return u.reshape(n, heads, size)

    base, dims = m["rot"]["base"], m["rot"]["dims"]
    return turn(make("q", H, d), base, dims, True), turn(make("k", G, d), base, dims, True), rms(make("v", G, e), eps)


def attend(q, k, v, scale: float, size: Optional[int], P: Optional[int], cap: Optional[float]) -> torch.Tensor:
    """q [n, H, d], k [n, G, d], v [n, G, e] -> [n, H, e]: tokens of the window and blocks before it in one softmax."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    vis = in_window(n, size)
    if P:
        k, v = torch.cat([k, pooled(k, P)]), torch.cat([v, pooled(v, P)])
        vis = torch.cat([vis, sees_block(n, size, P)], 1)
    kk, vv = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = capped(torch.einsum("ihd,jhd->hij", q, kk) * scale, cap)
    return torch.einsum("hij,jhe->ihe", softmax_over(s, vis), vv)


def window_attention(h, t, pre: str, m: dict, eps: float) -> torch.Tensor:
    q, k, v = projected(h, t, pre, m, eps)
    mask = m.get("mask") or {}
    out = attend(q, k, v, m["scale"], mask.get("size"), mask.get("pool"), m.get("softcap"))
    return (out * torch.sigmoid(h @ t[pre + "g"].T)[:, :, None]).reshape(h.shape[0], -1) @ t[pre + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------------------------
def choose_experts(z: torch.Tensor, correction: torch.Tensor, top: int):
    """z [n, E] router logits.  Returns (chosen [n, top] indices, weights [n, top])."""
    s = torch.softmax(z, -1)
    chosen = (s + correction).topk(top, dim=-1).indices
    return chosen, s.gather(1, chosen)


def expert_ff(h, t, pre: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    chosen, w = choose_experts(h @ t[pre + "router"].T, t[pre + "correction"], r["top"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        p = f"{pre}e{e}."
        for c in range(r["top"]):
            rows = (chosen[:, c] == e).nonzero()[:, 0]
            if len(rows):
                x = h[rows]
                out[rows] += w[rows, c][:, None] * ((silu(x @ t[p + "gate"].T) * (x @ t[p + "up"].T)) @ t[p + "down"].T)
    return out


# ---- the model ----------------------------------------------------------------------------------------------------------------
def forward(cfg: dict, t: Dict[str, torch.Tensor], tokens, dtype=torch.float64, taps: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of one sequence from position 0.  ``taps`` (a list) receives the stream after every layer."""
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in t.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kept: List[Optional[tuple]] = []
    for i, L in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", L["mixer"]
        h = norm(x, t[pre + "norm1"], eps)
        rows = None
        if L["type"] == "latent_attention":
            rows = kept[m["kv_from"]] if m.get("kv_from") is not None else latent_rows(h, t, pre + "mix.", m, eps)
            y = latent_attention(h, t, pre + "mix.", m, eps, rows)
        elif L["type"] == "retention":
            y = retention(h, t, pre + "mix.", m, eps)
        elif L["type"] == "attention":
            y = window_attention(h, t, pre + "mix.", m, eps)
        else:
            raise ValueError(L["type"])
        kept.append(rows)
        if L.get("mlp") is not None:
            y = y + expert_ff(h, t, pre + "mlp.", L["mlp"])
        x = x + mult * y
        if taps is not None:
            taps.append(x.clone())
    return norm(x, t["final.norm"], eps) @ t["head"].T
