"""A state-space memory with one fade per head and token (the Mamba-2 cell).

One projection makes ``[z | x | B | C | dt]`` of a token: z and x of ``num_heads`` heads of ``value_dim``, B and C
of ``groups`` groups of ``state_dim`` (head h reads group ``h // (num_heads / groups)``), dt one number per head.
x, B and C pass a short causal convolution over time per channel, with a bias, and silu.  Per head, with
``dt <- softplus(dt + dt_bias)``:

    S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T          y_t = S_t^T C_t + D x_t

y times silu(z) is RMS-normed in ``norm_groups`` equal parts with one weight over the row, and projected.

The walk is the one of linear attention (``csrc/linear_scan.cu``) with C for the query, B for the key, x for the
value and two numbers per token and head given from outside, exp(-exp(A_log) dt) and dt; prompt portions run
in chunks on the tensor cores where the sizes allow (``csrc/chunk_scan.cu``).  The projection leaves
its product in 32-bit; a kernel in front of the walk convolves and makes the two numbers, a kernel
behind it adds D x, gates and norms.  The state S and the convolution's last ``conv_taps - 1`` inputs are
32-bit ``StateSpec`` rows, zero when a request takes a slot.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import CompositeCacheSpec, ParamSpec, Part, StateSpec, register_mixer


@register_mixer("state_space")
class StateSpace(Part):
    graph_safe = True
    kernels = ("gemm", "state_space", "linear_scan")

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        s = spec
        if s.groups < 1 or s.num_heads % s.groups:
            raise ValueError(f"{s.num_heads} heads cannot share {s.groups} groups")
        if s.conv_taps < 1:
            raise ValueError(f"conv_taps must be at least 1, got {s.conv_taps}")
        self.inner, self.gn = s.num_heads * s.value_dim, s.groups * s.state_dim
        if s.norm_groups < 1 or self.inner % s.norm_groups:
            raise ValueError(f"{s.norm_groups} norm groups do not divide a row of {self.inner}")
        self.channels = self.inner + 2 * self.gn
        self.aligned = s.value_dim % 8 == 0 and s.state_dim % 8 == 0         # (16-byte rows of every operand)
        if self.aligned and rt.dtype == torch.bfloat16:
            self.kernels = self.kernels + ("chunk_scan",)

    @classmethod
    def params(cls, spec) -> Dict[str, ParamSpec]:
        H, n = spec.hidden_size, spec.num_heads
        inner, gn = n * spec.value_dim, spec.groups * spec.state_dim
        vec = dict(role="vector", init="normal")
        return {"in": ParamSpec((2 * inner + 2 * gn + n, H)), "conv": ParamSpec((inner + 2 * gn, spec.conv_taps), **vec),
                "conv_bias": ParamSpec((inner + 2 * gn,), **vec), "dt_bias": ParamSpec((n,), **vec), "A_log": ParamSpec((n,), **vec),
                "D": ParamSpec((n,), **vec), "norm": ParamSpec((inner,), role="vector", init="ones"), "o": ParamSpec((H, inner))}

    def load(self, tensors):
        w = tensors["in"]
        pad = -w.shape[0] % 8                       # rows of the product start on 16-byte boundaries: the columns behind dt are zero
        self.w_in = (torch.cat([w, w.new_zeros(pad, w.shape[1])]) if pad else w).contiguous()
        self.w_out = tensors["o"].contiguous()
        self.conv, self.conv_bias = tensors["conv"].contiguous(), tensors["conv_bias"].contiguous()
        self.dt_bias, self.a_log, self.d = (tensors[n].contiguous() for n in ("dt_bias", "A_log", "D"))
        self.norm = tensors["norm"].contiguous()
        self.skip = self.d.repeat_interleave(self.spec.value_dim).contiguous()        # (one number per channel, as the kernel reads it)

    def cache_spec(self):
        s = self.spec
        parts = [StateSpec((s.num_heads, s.value_dim, s.state_dim))]           # S, state channels contiguous
        if s.conv_taps > 1:
            parts.append(StateSpec((s.conv_taps - 1, self.channels)))          # the convolution's last inputs
        return CompositeCacheSpec(tuple(parts))

    def forward(self, x, ctx, cache, writes_cache: bool = True):
        s, ops = self.spec, self.rt.ops
        T, n, f32 = x.shape[0], s.num_heads, torch.float32
        x_off, dt_off = self.inner, self.inner + self.channels
        proj = ops.linear(x, self.w_in, out_dtype=f32)                        # [T, z | x | B | C | dt]
        u = self.rt.empty(T, self.channels)                                  # [T, x | B | C] convolved
        fades = self.rt.empty(3, T, n, dtype=f32)                            # keep, write, log keep
        conv_state = cache[1].state if s.conv_taps > 1 else None
        ops.state_space_prep(proj, x_off, dt_off, self.channels, self.conv, self.conv_bias, self.dt_bias, self.a_log, conv_state,
                             ctx, u, fades)
        y = self.rt.empty(T, self.inner, dtype=f32)
        first = ops.chunk_scan_first(ctx, self.rt.dtype, s.state_dim, s.value_dim) if self.aligned else None
        if first != 0:
            ops.linear_scan(u, self.inner + self.gn, self.inner, 0, n, s.state_dim, s.value_dim, "given", None, None, None, "none",
                            "none", "none", cache[0].state, ctx, y, keep=fades[0], write=fades[1], key_heads=s.groups,
                            requests=first)
        if first is not None:
            ops.chunk_scan(u, self.inner + self.gn, self.inner, 0, n, s.groups, s.state_dim, s.value_dim, cache[0].state, ctx, y,
                           first, log_keep=fades[2], write=fades[1])
        out = self.rt.empty(T, self.inner)
        ops.state_space_output(y, proj, x_off, u, self.skip, self.norm, n, s.norm_groups, s.eps, s.conv_taps, conv_state, ctx, out)
        return ops.linear(out, self.w_out)
