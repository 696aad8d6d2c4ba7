"""Linear attentions with a decay, per key channel or fixed per head, as mixers.

=============  ===========================  ==========================================
category       kind                         params
=============  ===========================  ==========================================
mixer          ``gated_linear_attention``   width, heads, head_dim (key channels of a
                                            head), v_dim, tau, eps, rank (of the decay's
                                            two-step projection; None: whatever the
                                            checkpoint's tensors have), q_scale (default
                                            head_dim^(-1/2)), names (q, k, v, gate, o,
                                            norm, decay_in, decay_out, decay_bias ->
                                            local names)
mixer          ``hgrn2``                    width, heads, head_dim (key channels of a
                                            head), v_dim, eps, names (q, forget,
                                            forget_bias, lower, v, norm, o -> local
                                            names)
mixer          ``retention``                width, heads, head_dim (key channels of a
                                            head), v_dim, decay (a number per head),
                                            eps, k_scale (default head_dim^(-1/2)),
                                            position (PartSpec ``rotary_pairs`` of
                                            pairing ``halves``, or None), names (q, k,
                                            v, gate, o -> local names)
=============  ===========================  ==========================================

``gated_linear_attention``, with h the mixer's input, H heads of dk key channels and dv value numbers:

* q = Wq h * q_scale, k = Wk h (H x dk each), v = Wv h (H x dv), g = Wg h (H x dv), low = W1 h (r numbers): one matrix
  product;
* z = W2 low + b (H x dk numbers); the decay of a key channel is a = sigmoid(z)^(1 / tau), evaluated as
  exp(-softplus(-z) / tau);
* per head S <- diag(a) S + k v^T (dk x dv; the decay acts on the rows that belong to key channels), o = S^T q;
* every head's o is divided by its root mean square over dv (eps inside the root) and multiplied by a weight of dv numbers
  that the heads share; the heads side by side are multiplied by silu(g) and go through Wo.

``hgrn2``, with the same letters:

* q = silu(Wq h), z = Wf h + b (H x dk each), v = Wv h (H x dv): one matrix product;
* the forget factor of a key channel is f = l + (1 - l) sigmoid(z), l the channel's learned lower bound;
* per head S <- diag(f) S + (1 - f) v^T, o = S^T q: the recurrence above with the decay f and 1 - f (evaluated as
  (1 - l) sigmoid(-z)) where it has a key;
* the per-head norm above, no gate, Wo.

``retention``, with the same letters:

* q = Wq h, k = Wk h (H x dk each), v = Wv h (H x dv), g = Wg h (H x dv): one matrix product; the position encoding turns q
  and k, k is multiplied by ``k_scale`` afterwards;
* per head S <- a S + k v^T with the head's fixed number a, o = S^T q;
* every head's o is divided by its root mean square (no weight); the heads side by side are multiplied by silu(g) and go
  through Wo.

The state is one float32 record per sequence (kind ``state`` of the cache: zero when a sequence starts), read and brought
up to date by every step whatever its shape.  Everything between the two matrix products is float32, W2's product
included (W2 is held in float32; its rank is small).
"""
from __future__ import annotations

import torch

from .. import ops
from ..models.spec import PartSpec
from .attention import RotaryPairs
from .base import CacheNeed, Mixer, TensorSpec, build_part, register_part
from .linear import Linear
from .standard import NoPosition


class GatedLinearAttention(Mixer):
    PROMPT_CAPTURABLE = True
    RANDOM_RANK = 16                      # the rank random weights are drawn with where the parameters leave it open

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        p = params
        self.width, self.heads = int(p["width"]), int(p["heads"])
        self.key_dim, self.v_dim = int(p["head_dim"]), int(p["v_dim"])
        self.tau, self.eps = float(p["tau"]), float(p["eps"])
        if self.heads <= 0 or self.key_dim <= 0 or self.v_dim <= 0 or self.tau <= 0:
            raise ValueError("heads, head_dim, v_dim and tau must be positive")
        self.rank = int(p["rank"]) if p.get("rank") else None
        self.q_scale = float(p["q_scale"]) if p.get("q_scale") is not None else self.key_dim ** -0.5
        self.hk, self.hv = self.heads * self.key_dim, self.heads * self.v_dim
        names = dict(q="q_proj.weight", k="k_proj.weight", v="v_proj.weight", gate="g_proj.weight", o="o_proj.weight",
                     norm="norm.weight", decay_in="decay_in.weight", decay_out="decay_out.weight", decay_bias="decay_out.bias")
        names.update(p.get("names") or {})
        self.names = names
        self.input = None                 # Linear over [q | k | v | g | low]; made when the rank is known
        self.o = Linear(self.width, self.hv, ctx)
        self.w2 = self.b2 = self.norm_w = None

    def tensor_specs(self):
        nm, r = self.names, (self.rank if self.rank is not None else -1)
        return [TensorSpec(nm["q"], (self.hk, self.width)), TensorSpec(nm["k"], (self.hk, self.width)),
                TensorSpec(nm["v"], (self.hv, self.width)), TensorSpec(nm["gate"], (self.hv, self.width)),
                TensorSpec(nm["o"], (self.width, self.hv)), TensorSpec(nm["norm"], (self.v_dim,), "vector"),
                TensorSpec(nm["decay_in"], (r, self.width), init_arg=self.RANDOM_RANK),
                TensorSpec(nm["decay_out"], (self.hk, r), "vector", init="decay_out", init_arg=self.RANDOM_RANK),
                TensorSpec(nm["decay_bias"], (self.hk,), "vector", init="decay_bias")]

    def load(self, fetch):
        nm, hold = self.names, self.ctx.hold
        low, w2 = fetch(nm["decay_in"]), fetch(nm["decay_out"])
        rank = int(low.shape[0])
        if rank <= 0 or tuple(w2.shape) != (self.hk, rank) or (self.rank is not None and rank != self.rank):
            raise ValueError(f"the decay's projections have shapes {tuple(low.shape)} and {tuple(w2.shape)}; "
                             f"[r, {self.width}] and [{self.hk}, r] with one r are expected")
        self.loaded_rank = rank
        self.input = Linear(2 * self.hk + 2 * self.hv + rank, self.width, self.ctx)
        self.input.load_rows([fetch(nm["q"]), fetch(nm["k"]), fetch(nm["v"]), fetch(nm["gate"]), low])
        self.o.load_rows([fetch(nm["o"])])
        # (a matrix of the checkpoint's 16-bit numbers is the same numbers in float32)
        self.w2, self.b2 = hold(w2, "vector"), hold(fetch(nm["decay_bias"]), "vector")
        self.norm_w = hold(fetch(nm["norm"]), "vector")

    def tensor(self, name):
        nm, hk, hv = self.names, self.hk, self.hv
        spans = {nm["q"]: (0, hk), nm["k"]: (hk, 2 * hk), nm["v"]: (2 * hk, 2 * hk + hv), nm["gate"]: (2 * hk + hv, 2 * hk + 2 * hv)}
        if self.input is not None and name in spans:
            return self.input.rows(*spans[name])
        if self.input is not None and name == nm["decay_in"]:
            return self.input.rows(2 * hk + 2 * hv, 2 * hk + 2 * hv + self.loaded_rank)
        if name == nm["o"]:
            return self.o.rows(0, self.width)
        return {nm["decay_out"]: self.w2, nm["decay_bias"]: self.b2, nm["norm"]: self.norm_w}.get(name)

    def record_floats(self) -> int:
        return self.hv * self.key_dim

    def cache_need(self):
        return CacheNeed("state", shape=(self.record_floats(),), dtype=torch.float32)

    def weight_bytes(self):
        n = self.o.weight_bytes() + (self.input.weight_bytes() if self.input is not None else 0)
        return n + 4 * (self.hk * (1 + (self.loaded_rank if self.input is not None else 0)) + self.v_dim)

    def forward(self, x, batch, cache, write_cache):
        if not write_cache:
            raise RuntimeError("a linear-attention mixer keeps its own record; it cannot read another entry's")
        parts = self.input.forward_delta(x)                         # float32 [splits, n, cols]
        y = ops.gla_mix(parts, heads=self.heads, key_dim=self.key_dim, v_dim=self.v_dim, w2=self.w2, b2=self.b2, q_scale=self.q_scale,
                        tau=self.tau, records=cache.state, batch=batch)
        g = ops.gla_norm_gate(y, parts, 2 * self.hk + self.hv, self.heads, self.v_dim, self.norm_w, self.eps, self.ctx.dtype)
        return self.o.forward_delta(g)


class Hgrn2(Mixer):
    PROMPT_CAPTURABLE = True

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        p = params
        self.width, self.heads = int(p["width"]), int(p["heads"])
        self.key_dim, self.v_dim, self.eps = int(p["head_dim"]), int(p["v_dim"]), float(p["eps"])
        if self.heads <= 0 or self.key_dim <= 0 or self.v_dim <= 0:
            raise ValueError("heads, head_dim and v_dim must be positive")
        self.hk, self.hv = self.heads * self.key_dim, self.heads * self.v_dim
        names = dict(q="q_proj.weight", forget="f_proj.weight", forget_bias="f_proj.bias", lower="lower_bound", v="v_proj.weight",
                     norm="norm.weight", o="o_proj.weight")
        names.update(p.get("names") or {})
        self.names = names
        self.input = Linear(2 * self.hk + self.hv, self.width, ctx)          # rows: q, forget, v
        self.o = Linear(self.width, self.hv, ctx)
        self.bias = self.lower = self.norm_w = None

    def tensor_specs(self):
        nm = self.names
        return [TensorSpec(nm["q"], (self.hk, self.width)), TensorSpec(nm["forget"], (self.hk, self.width)),
                TensorSpec(nm["forget_bias"], (self.hk,), "vector", init="decay_bias"),
                TensorSpec(nm["lower"], (self.hk,), "vector", init="unit_interval"), TensorSpec(nm["v"], (self.hv, self.width)),
                TensorSpec(nm["norm"], (self.v_dim,), "vector"), TensorSpec(nm["o"], (self.width, self.hv))]

    def load(self, fetch):
        nm, hold = self.names, self.ctx.hold
        self.input.load_rows([fetch(nm["q"]), fetch(nm["forget"]), fetch(nm["v"])])
        self.o.load_rows([fetch(nm["o"])])
        self.bias, self.lower, self.norm_w = (hold(fetch(nm[k]), "vector") for k in ("forget_bias", "lower", "norm"))

    def tensor(self, name):
        nm, hk = self.names, self.hk
        spans = {nm["q"]: (0, hk), nm["forget"]: (hk, 2 * hk), nm["v"]: (2 * hk, 2 * hk + self.hv)}
        if name in spans:
            return self.input.rows(*spans[name])
        if name == nm["o"]:
            return self.o.rows(0, self.width)
        return {nm["forget_bias"]: self.bias, nm["lower"]: self.lower, nm["norm"]: self.norm_w}.get(name)

    def record_floats(self) -> int:
        return self.hv * self.key_dim

    def cache_need(self):
        return CacheNeed("state", shape=(self.record_floats(),), dtype=torch.float32)

    def weight_bytes(self):
        return self.input.weight_bytes() + self.o.weight_bytes() + 4 * (2 * self.hk + self.v_dim)

    def forward(self, x, batch, cache, write_cache):
        if not write_cache:
            raise RuntimeError("a linear-attention mixer keeps its own record; it cannot read another entry's")
        parts = self.input.forward_delta(x)                         # float32 [splits, n, 2 H dk + H dv]
        y = ops.hgrn2_mix(parts, heads=self.heads, key_dim=self.key_dim, v_dim=self.v_dim, bias=self.bias, lower=self.lower,
                          records=cache.state, batch=batch)
        g = ops.gla_norm_gate(y, None, 0, self.heads, self.v_dim, self.norm_w, self.eps, self.ctx.dtype)
        return self.o.forward_delta(g)


register_part("mixer", "gated_linear_attention", GatedLinearAttention)
class Retention(Mixer):
    PROMPT_CAPTURABLE = True

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        p = params
        self.width, self.heads = int(p["width"]), int(p["heads"])
        self.key_dim, self.v_dim, self.eps = int(p["head_dim"]), int(p["v_dim"]), float(p["eps"])
        decay = [float(a) for a in p["decay"]]
        if self.heads <= 0 or self.key_dim <= 0 or self.v_dim <= 0 or len(decay) != self.heads:
            raise ValueError("heads, head_dim and v_dim must be positive, and every head has a decay")
        self.decay = torch.tensor(decay, dtype=torch.float32, device=ctx.device)
        self.k_scale = float(p["k_scale"]) if p.get("k_scale") is not None else self.key_dim ** -0.5
        self.position = build_part("position", p.get("position") or PartSpec("none"), ctx)
        if not isinstance(self.position, NoPosition) and not (
                isinstance(self.position, RotaryPairs) and self.position.pairing == "halves" and self.position.head_dim == self.key_dim):
            raise ValueError("this mixer's kernel turns half-split pairs (rotary_pairs) of its heads or nothing")
        self.hk, self.hv = self.heads * self.key_dim, self.heads * self.v_dim
        names = dict(q="q_proj.weight", k="k_proj.weight", v="v_proj.weight", gate="g_proj.weight", o="o_proj.weight")
        names.update(p.get("names") or {})
        self.names = names
        self.input = Linear(2 * self.hk + 2 * self.hv, self.width, ctx)      # rows: q, k, v, gate
        self.o = Linear(self.width, self.hv, ctx)

    def tensor_specs(self):
        nm = self.names
        return [TensorSpec(nm["q"], (self.hk, self.width)), TensorSpec(nm["k"], (self.hk, self.width)),
                TensorSpec(nm["v"], (self.hv, self.width)), TensorSpec(nm["gate"], (self.hv, self.width)),
                TensorSpec(nm["o"], (self.width, self.hv))]

    def load(self, fetch):
        nm = self.names
        self.input.load_rows([fetch(nm[k]) for k in ("q", "k", "v", "gate")])
        self.o.load_rows([fetch(nm["o"])])

    def tensor(self, name):
        nm, hk, hv = self.names, self.hk, self.hv
        spans = {nm["q"]: (0, hk), nm["k"]: (hk, 2 * hk), nm["v"]: (2 * hk, 2 * hk + hv), nm["gate"]: (2 * hk + hv, 2 * hk + 2 * hv)}
        if name in spans:
            return self.input.rows(*spans[name])
        return self.o.rows(0, self.width) if name == nm["o"] else None

    def record_floats(self) -> int:
        return self.hv * self.key_dim

    def cache_need(self):
        return CacheNeed("state", shape=(self.record_floats(),), dtype=torch.float32)

    def weight_bytes(self):
        return self.input.weight_bytes() + self.o.weight_bytes()

    def forward(self, x, batch, cache, write_cache):
        if not write_cache:
            raise RuntimeError("a linear-attention mixer keeps its own record; it cannot read another entry's")
        parts = self.input.forward_delta(x)                         # float32 [splits, n, 2 H dk + 2 H dv]
        rot = self.position if isinstance(self.position, RotaryPairs) else None
        cos, sin = rot.tables(batch) if rot else (None, None)
        y = ops.retention_mix(parts, heads=self.heads, key_dim=self.key_dim, v_dim=self.v_dim, cos=cos, sin=sin, rot_dims=rot.dims if rot else 0,
                              k_scale=self.k_scale, decay=self.decay, records=cache.state, batch=batch)
        g = ops.gla_norm_gate(y, parts, 2 * self.hk + self.hv, self.heads, self.v_dim, None, self.eps, self.ctx.dtype)
        return self.o.forward_delta(g)


register_part("mixer", "hgrn2", Hgrn2)
register_part("mixer", "retention", Retention)
