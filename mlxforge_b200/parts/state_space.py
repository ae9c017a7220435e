"""State-space mixers: recurrences whose decay and step size depend on the token.

``mamba2``: one projection of the input is cut into a gate ``z``, values ``x`` (``n_heads`` heads of ``head_dim``),
``B`` and ``C`` (``n_groups`` groups of ``state``) and a step-size logit per head.  x, B and C together pass a short
causal convolution over time per channel (``conv`` taps with a bias, the last tap the current token's, zeros
before the start) and SiLU.  Per head (head h reads group ``h // (n_heads / n_groups)``), with a 32-bit state
``S`` [state, head_dim] per request:

    dt = softplus(logit + dt_bias_h) ;  S <- exp(-exp(A_log_h) dt) S + dt B x^T ;  y = S^T C + D_h x

The heads' read-outs are concatenated, multiplied by ``silu(z)``, divided by their root mean square in
``norm_groups`` equal parts, multiplied by a plain weight and projected.

``selective_scan``: ``[x | z] = W_in h`` (``inner`` channels each), x through such a convolution and SiLU, then
``[dt_low | B | C] = W_x x`` and one step-size logit per channel, ``W_dt dt_low + bias``.  Per channel c and state n:

    dt_c = softplus(.) ;  S[c, n] <- exp(-exp(A_log[c, n]) dt_c) S[c, n] + dt_c x_c B_n ;
    y_c = sum_n S[c, n] C_n + D_c x_c

and the output is ``W_o (y * silu(z))``.

A request's slot keeps ``S`` and the last ``conv - 1`` inputs of the convolution, so a step goes on from where
the step before ended, however the prompt was cut.  Projections that read one input are one product, written in
32-bit; what follows is 32-bit.  Long portions are cut into segments that run side by side (``scan_min_tokens``,
the least length of one); ``names`` maps the tensors' roles to their names."""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from .base import FixedState, Mixer, TensorSpec, register_mixer


def pad4(n: int) -> int:
    """State sizes in whole pieces of 16 bytes, so that every part of a slot starts on one."""
    return (n + 3) // 4 * 4


class _Scan(Mixer):
    """What the mixers with a linear recurrence share: names, segments and their scratch."""

    graph_safe = True
    roles: Dict[str, str] = {}

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.hidden = int(params["hidden_size"])
        self.out_f32 = bool(params.get("out_f32", False))
        self.min_tokens = int(params.get("scan_min_tokens", 64))
        if self.min_tokens < 1:
            raise ValueError("scan_min_tokens must be at least 1")
        self.names = dict(self.roles, **(params.get("names") or {}))

    def _n(self, role: str) -> str:
        return self.prefix + self.names[role]

    def _segments(self, batch, blocks: int, residents, state_floats: int, decay_floats: int):
        seg = ops.scan_segments(batch, blocks, residents, state_floats, self.min_tokens)
        if seg[0] == 1:
            return seg, None
        n = batch.n_seqs * seg[0]
        return seg, (self.rt.buffer("scan.seg_state", (n * state_floats,), torch.float32),
                     self.rt.buffer("scan.seg_decay", (n * decay_floats,), torch.float32))

    def _readouts(self, T: int, parts: int, width: int):
        return self.rt.buffer("scan.o", (T, parts * width), torch.float32).view(parts, T, width)

    def _out(self, y, w):
        return self.rt.linear(y, w, self.rt.buffer("scan.delta", (y.shape[0], self.hidden),
                                                   torch.float32 if self.out_f32 else None))


@register_mixer("mamba2")
class Mamba2(_Scan):
    roles = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D",
             "norm": "norm", "o": "o"}

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        p = params
        self.n_heads, self.vdim, self.state = int(p["n_heads"]), int(p["head_dim"]), int(p["state"])
        self.groups, self.norm_groups = int(p.get("n_groups", 1)), int(p.get("norm_groups", 1))
        self.taps, self.eps = int(p["conv"]), float(p["eps"])
        self.inner = self.n_heads * self.vdim
        self.bc = self.groups * self.state
        self.channels = self.inner + 2 * self.bc
        if self.groups < 1 or self.n_heads % self.groups:
            raise ValueError("mamba2: n_heads must be a multiple of n_groups")
        if self.norm_groups < 1 or self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.inner} channels do not divide into {self.norm_groups} norm groups")
        if self.taps < 1:
            raise ValueError("mamba2: conv must be at least 1 tap")
        self.state_floats = self.n_heads * self.state * self.vdim
        self.conv_off = pad4(self.state_floats)
        self.width = self.inner + self.channels + self.n_heads
        self.w_in = self.w_o = self.conv_w = self.conv_b = self.dt_bias = self.a_log = self.d = self.norm_w = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        nh, C = self.n_heads, self.channels
        return {self._n("in"): TensorSpec((self.width, self.hidden)),
                self._n("conv"): TensorSpec((C, self.taps), role="vector"),
                self._n("conv_bias"): TensorSpec((C,), role="vector"),
                self._n("dt_bias"): TensorSpec((nh,), role="vector"), self._n("A_log"): TensorSpec((nh,), role="vector"),
                self._n("D"): TensorSpec((nh,), role="vector"), self._n("norm"): TensorSpec((self.inner,), role="vector"),
                self._n("o"): TensorSpec((self.hidden, self.inner))}

    def bind(self, tensors) -> None:
        dt, f32 = self.rt.dtype, torch.float32
        w = tensors[self._n("in")].to(dt)
        pad = pad4(self.width) - self.width
        if pad:                                    # rows of the projection in whole pieces of 16 bytes
            w = torch.cat([w, torch.zeros((pad, self.hidden), dtype=dt, device=w.device)], dim=0)
        self.w_in = w.contiguous()
        self.w_o = tensors[self._n("o")].to(dt).contiguous()
        vec = lambda r: tensors[self._n(r)].to(f32).contiguous()
        self.conv_w, self.conv_b, self.dt_bias, self.a_log = vec("conv"), vec("conv_bias"), vec("dt_bias"), vec("A_log")
        self.d, self.norm_w = vec("D"), vec("norm")

    def weight_bytes(self) -> int:
        return (self.w_in.numel() + self.w_o.numel()) * self.w_in.element_size()

    def cache_need(self):
        return FixedState((pad4(self.conv_off + (self.taps - 1) * self.channels),), tag="mamba2")

    def forward(self, x, batch, cache, writes_cache: bool = True):
        rt, T, f32 = self.rt, x.shape[0], torch.float32
        proj = rt.linear(x, self.w_in, rt.buffer("mamba2.in", (T, self.w_in.shape[0]), f32))
        ld = proj.shape[1]
        xbc = rt.buffer("mamba2.xbc", (T, self.channels), f32)
        ops.conv_act(proj[:, self.inner:], ld, self.conv_w, self.conv_b, True, cache.tensor, self.conv_off, batch, xbc)
        o = self._readouts(T, ops.decay_parts(self.state, self.vdim), self.inner)
        seg, scratch = self._segments(batch, ops.decay_blocks(self.n_heads, self.state, self.vdim),
                                      ops.decay_residents(self.state, self.vdim, False), self.state_floats, self.n_heads)
        C = self.channels
        ops.decay_recurrence(xbc[:, self.inner + self.bc:], C, xbc[:, self.inner:], C, xbc, C, cache.tensor, batch, o,
                             self.n_heads, self.groups, self.state, self.vdim, dt=proj[:, self.inner + C:], dt_ld=ld,
                             dt_bias=self.dt_bias, a_log=self.a_log, skip=self.d, segments=seg, scratch=scratch)
        y = rt.buffer("scan.y", (T, self.inner))
        ops.gated_norm(o, proj, ld, self.norm_w, self.eps, y, self.norm_groups, True)
        return self._out(y, self.w_o)


@register_mixer("selective_scan")
class SelectiveScan(_Scan):
    roles = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "x": "x", "dt": "dt", "dt_bias": "dt.b", "A_log": "A_log",
             "D": "D", "o": "o"}

    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        p = params
        self.inner, self.state, self.rank = int(p["inner"]), int(p["state"]), int(p["dt_rank"])
        self.taps = int(p["conv"])
        if self.taps < 1 or self.rank < 1:
            raise ValueError("selective_scan: conv and dt_rank must be at least 1")
        if self.state > 512:
            raise ValueError(f"selective_scan: {self.state} states per channel are more than the kernel's 512")
        self.state_floats = self.inner * self.state
        self.conv_off = pad4(self.state_floats)
        # tokens and rank from which the step-size logits are a product instead of the narrow kernel's
        self.product_min_tokens, self.product_min_rank = 65, 32
        self.w_in = self.w_x = self.w_dt = self.w_dt_t = self.w_o = None
        self.conv_w = self.conv_b = self.dt_bias = self.a = self.d = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        n, H = self.inner, self.hidden
        return {self._n("in"): TensorSpec((2 * n, H)), self._n("conv"): TensorSpec((n, self.taps), role="vector"),
                self._n("conv_bias"): TensorSpec((n,), role="vector"),
                self._n("x"): TensorSpec((self.rank + 2 * self.state, n)), self._n("dt"): TensorSpec((n, self.rank)),
                self._n("dt_bias"): TensorSpec((n,), role="vector"),
                self._n("A_log"): TensorSpec((n, self.state), role="vector"), self._n("D"): TensorSpec((n,), role="vector"),
                self._n("o"): TensorSpec((H, n))}

    def bind(self, tensors) -> None:
        dt, f32 = self.rt.dtype, torch.float32
        mat = lambda r: tensors[self._n(r)].to(dt).contiguous()
        vec = lambda r: tensors[self._n(r)].to(f32).contiguous()
        self.w_in, self.w_x, self.w_dt, self.w_o = mat("in"), mat("x"), mat("dt"), mat("o")
        self.w_dt_t = self.w_dt.t().contiguous()
        self.conv_w, self.conv_b, self.dt_bias, self.d = vec("conv"), vec("conv_bias"), vec("dt_bias"), vec("D")
        self.a = (-torch.exp(tensors[self._n("A_log")].to(torch.float64))).to(f32).contiguous()

    def weight_bytes(self) -> int:
        return (self.w_in.numel() + self.w_x.numel() + self.w_dt.numel() + self.w_o.numel()) * self.w_in.element_size()

    def cache_need(self):
        return FixedState((pad4(self.conv_off + (self.taps - 1) * self.inner),), tag="selective_scan")

    def forward(self, x, batch, cache, writes_cache: bool = True):
        rt, T, f32, n, R = self.rt, x.shape[0], torch.float32, self.inner, self.rank
        proj = rt.linear(x, self.w_in, rt.buffer("sscan.in", (T, 2 * n), f32))
        u = rt.buffer("sscan.u", (T, n), f32)
        u16 = None if rt.dtype == f32 else rt.buffer("sscan.u16", (T, n))        # for the product that reads it
        ops.conv_act(proj, 2 * n, self.conv_w, self.conv_b, True, cache.tensor, self.conv_off, batch, u, u16)
        low = rt.linear(u if u16 is None else u16, self.w_x, rt.buffer("sscan.low", (T, R + 2 * self.state), f32))
        dt = rt.buffer("sscan.dt", (T, n), f32)
        if T >= self.product_min_tokens and R >= self.product_min_rank:
            dt_low = rt.buffer("sscan.dt_low", (T, R))
            dt_low.copy_(low[:, :R])
            rt.linear(dt_low, self.w_dt, dt)
        else:
            ops.low_rank(low, low.shape[1], self.w_dt_t, None, dt)
        seg, scratch = self._segments(batch, ops.scan_blocks(n, self.state), ops.scan_residents(self.state), self.state_floats, n)
        y = rt.buffer("sscan.y", (T, n))
        ops.selective_scan(u, dt, n, self.dt_bias, proj[:, n:], 2 * n, low[:, R:], low.shape[1], self.a, self.d,
                           cache.tensor, batch, y, self.state, seg, scratch)
        return rt.linear(y, self.w_o, rt.buffer("sscan.delta", (T, self.hidden), f32 if self.out_f32 else None))
