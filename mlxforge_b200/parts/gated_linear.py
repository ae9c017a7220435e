"""Gated linear attention: a linear recurrence with a decay per key channel that depends on the token.

Per head, with a 32-bit state ``S`` [head_dim, v_head_dim] per request that starts at zero, token after token:

    S <- diag(alpha_t) S + k_t v_t^T ;   o_t = S^T q_t ;   alpha_t = sigmoid(W_a2 (W_a1 h) + bias)^(1 / tau)

``q`` (times ``head_dim^-1/2``), ``k`` (``n_heads`` heads of ``head_dim``) and ``v`` (``n_heads`` heads of ``v_head_dim``) are
projections of the input.  Every head's read-out is divided by its root mean square over ``v_head_dim`` (``eps``),
multiplied by a plain weight shared by the heads; the heads are concatenated, multiplied by ``silu(W_g h)`` and
projected by ``W_o``.

All projections that read the input are one product, written in 32-bit; the narrow second factor of the decay
and the decay itself are one kernel; everything after the projections is 32-bit.  The request's slot keeps
``S``.  ``names`` maps the tensors' roles to their names."""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from .base import FixedState, TensorSpec, register_mixer
from .state_space import _Scan, pad4


@register_mixer("gated_linear")
class GatedLinear(_Scan):
    roles = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "a1": "a1", "a2": "a2", "a_bias": "a2.b"}

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        p = params
        self.n_heads, self.dim = int(p["n_heads"]), int(p["head_dim"])
        self.vdim = int(p.get("v_head_dim") or self.dim)
        self.rank, self.tau, self.eps = int(p["decay_rank"]), float(p["tau"]), float(p["eps"])
        self.q_scale = float(p.get("query_scale", self.dim ** -0.5))
        if self.rank < 1 or not self.tau > 0:
            raise ValueError("gated_linear: decay_rank must be at least 1 and tau positive")
        self.state_floats = self.n_heads * self.dim * self.vdim
        self.w_in = self.w_a2_t = self.a_bias = self.w_o = self.norm_w = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        nqk, nv, H = self.n_heads * self.dim, self.n_heads * self.vdim, self.hidden
        rows = {"q": nqk, "k": nqk, "v": nv, "g": nv, "a1": self.rank}
        specs = {self._n(r): TensorSpec((n, H)) for r, n in rows.items()}
        specs.update({self._n("o"): TensorSpec((H, nv)), self._n("norm"): TensorSpec((self.vdim,), role="vector"),
                      self._n("a2"): TensorSpec((nqk, self.rank)), self._n("a_bias"): TensorSpec((nqk,), role="vector")})
        return specs

    def bind(self, tensors) -> None:
        dt, f32 = self.rt.dtype, torch.float32
        rows = [tensors[self._n(r)].to(dt) for r in ("q", "k", "v", "g", "a1")]
        n = sum(r.shape[0] for r in rows)
        if pad4(n) != n:                           # rows of the projection in whole pieces of 16 bytes
            rows.append(torch.zeros((pad4(n) - n, self.hidden), dtype=dt, device=rows[0].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_a2_t = tensors[self._n("a2")].to(dt).t().contiguous()
        self.w_o = tensors[self._n("o")].to(dt).contiguous()
        self.a_bias = tensors[self._n("a_bias")].to(f32).contiguous()
        self.norm_w = tensors[self._n("norm")].to(f32).contiguous()

    def weight_bytes(self) -> int:
        return (self.w_in.numel() + self.w_a2_t.numel() + self.w_o.numel()) * self.w_in.element_size()

    def cache_need(self):
        return FixedState((pad4(self.state_floats),), tag="gated_linear")

    def forward(self, x, batch, cache, writes_cache: bool = True):
        rt, T, f32, nh, d, dv = self.rt, x.shape[0], torch.float32, self.n_heads, self.dim, self.vdim
        proj = rt.linear(x, self.w_in, rt.buffer("gla.in", (T, self.w_in.shape[0]), f32))
        ld, nqk, nv = proj.shape[1], nh * d, nh * dv
        alpha = rt.buffer("gla.alpha", (T, nqk), f32)
        ops.low_rank(proj[:, 2 * nqk + 2 * nv:], ld, self.w_a2_t, self.a_bias, alpha, decay_tau=self.tau)
        o = self._readouts(T, ops.decay_parts(d, dv), nv)
        seg, scratch = self._segments(batch, ops.decay_blocks(nh, d, dv), ops.decay_residents(d, dv, True), self.state_floats, nqk)
        ops.decay_recurrence(proj, ld, proj[:, nqk:], ld, proj[:, 2 * nqk:], ld, cache.tensor, batch, o, nh, nh, d, dv,
                             alpha=alpha, q_scale=self.q_scale, segments=seg, scratch=scratch)
        y = rt.buffer("scan.y", (T, nv))
        ops.gated_norm(o, proj[:, 2 * nqk + nv:], ld, self.norm_w, self.eps, y, nh, False)
        return self._out(y, self.w_o)
