"""Linear attention with a matrix state per head and request.

Per head, with q and the write vector b of ``key_dim`` channels and v of ``value_dim``:

    S_t = diag(a_t) S_(t-1) + b_t v_t^T          o_t = S_t^T q_t

The spec's ``gate`` says where a and b come from: one constant per head and a key projection
("fixed_decay": S decays uniformly, b = act(W_k x)), or a forget gate per channel with a learnt
floor that also sets the write strength ("forget": a = floor + (1 - floor) sigmoid(W_f x + bias),
b = 1 - a; no key, no other scale).  The outputs are RMS-normed (all heads together with one weight
over the row, or each head by itself with one weight of head size or none), optionally multiplied by
sigmoid or silu of W_g x, and projected by W_o.  With a fixed decay q and k may be rotated by the tokens'
positions and k scaled (retention): the projections leave their product in 32-bit, walked tokens are rotated
there, and prompt portions run in chunks on the tensor cores (``csrc/chunk_scan.cu``) with rotated queries and
keys as sums of two bfloat16 numbers.

The state starts at zero when a request takes a slot, is 32-bit, and is carried from step to
step in the slot's row of a ``StateSpec`` cache.  One product makes all projections of a step
(rows of W_q, then W_k or W_f, then W_v, then W_g), one kernel walks every request's tokens in
order (prompt portions and single tokens alike), one kernel norms and gates.  Gates, decays, the
state and the norm are 32-bit whatever the compute dtype.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import POSITIONS, ParamSpec, Part, StateSpec, register_mixer


@register_mixer("linear_recurrence")
class LinearRecurrence(Part):
    graph_safe = True
    kernels = ("gemm", "linear_scan", "rownorm")

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        s = spec
        if s.gate not in ("fixed_decay", "forget"):
            raise ValueError(f"gate '{s.gate}' is not known (fixed_decay, forget)")
        if s.gate == "fixed_decay" and len(s.decay) != s.num_heads:
            raise ValueError(f"{len(s.decay)} decays for {s.num_heads} heads")
        if s.out_norm not in ("all", "per_head", "unit"):
            raise ValueError(f"out_norm '{s.out_norm}' is not known (all, per_head, unit)")
        self.gate_act = getattr(s, "out_gate_activation", "sigmoid")
        if self.gate_act not in ("sigmoid", "silu"):
            raise ValueError(f"out_gate_activation '{self.gate_act}' is not known (sigmoid, silu)")
        position = getattr(s, "position", None)
        self.position = POSITIONS.build(position, rt) if position is not None and position.kind != "none" else None
        self.table = self.position.rotary_table() if self.position is not None else None
        if self.position is not None and (self.table is None or getattr(position, "pairing", "half") != "half"
                                          or s.gate != "fixed_decay" or s.q_activation != "none" or s.k_activation != "none"):
            raise ValueError("a rotation of q and k is in halves and goes with a fixed decay, without activations on q and k")
        self.k_scale = float(getattr(s, "k_scale", 1.0))
        if self.k_scale != 1.0 and s.gate != "fixed_decay":
            raise ValueError("a factor on k goes with a fixed decay")
        if self.position is not None and rt.dtype == torch.bfloat16:
            self.kernels = self.kernels + ("chunk_scan",)
        # the output kernel that knows heads without a weight and the silu gate
        self.plain_output = s.out_norm != "unit" and self.gate_act == "sigmoid"
        if not self.plain_output:
            self.kernels = self.kernels + ("delta_rule",)
        for a in (s.q_activation, s.k_activation, s.v_activation):
            if a not in ("none", "silu"):
                raise ValueError(f"activation '{a}' is not implemented here (none, silu)")
        self.qk = s.num_heads * s.key_dim
        self.vv = s.num_heads * s.value_dim
        self.decay = self.log_decay = None
        if s.gate == "fixed_decay":
            decay = torch.tensor([float(d) for d in s.decay], dtype=torch.float64)
            self.decay = decay.to(dtype=torch.float32, device=rt.device)
            if bool((decay >= 0).all()):
                self.log_decay = torch.log(decay).to(dtype=torch.float32, device=rt.device)

    @classmethod
    def params(cls, spec) -> Dict[str, ParamSpec]:
        H = spec.hidden_size
        qk, vv = spec.num_heads * spec.key_dim, spec.num_heads * spec.value_dim
        p = {"q": ParamSpec((qk, H)), "v": ParamSpec((vv, H)), "o": ParamSpec((H, vv))}
        if spec.gate == "fixed_decay":
            p["k"] = ParamSpec((qk, H))
        else:
            p["f"] = ParamSpec((qk, H))
            p["f_bias"] = ParamSpec((qk,), role="vector", init="normal")
            p["floor"] = ParamSpec((qk,), role="vector", init="normal")
        if spec.out_gate:
            p["g"] = ParamSpec((vv, H))
        if spec.out_norm == "unit":
            return p
        p["norm"] = ParamSpec((vv if spec.out_norm == "all" else spec.value_dim,), role="vector", init="ones")
        return p

    def load(self, tensors):
        s = self.spec
        second = tensors["k"] if s.gate == "fixed_decay" else tensors["f"]
        rows = [tensors["q"], second, tensors["v"]] + ([tensors["g"]] if s.out_gate else [])
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_out = tensors["o"].contiguous()
        self.norm = tensors.get("norm")
        self.f_bias = tensors.get("f_bias")
        self.floor = tensors.get("floor")

    def cache_spec(self):
        s = self.spec
        return StateSpec((s.num_heads, s.value_dim, s.key_dim))     # key channels contiguous

    def _walk(self, proj, ctx, cache, o, **extra):
        s = self.spec
        if self.k_scale != 1.0:                     # (a factor on k is one on the read-out: it rides on q)
            extra["q_scale"] = self.k_scale
        self.rt.ops.linear_scan(proj, 0, self.qk, 2 * self.qk, s.num_heads, s.key_dim, s.value_dim, s.gate,
                                self.decay, self.f_bias, self.floor, s.q_activation, s.k_activation, s.v_activation,
                                cache.state, ctx, o, **extra)

    def forward(self, x, ctx, cache, writes_cache: bool = True):
        s, ops = self.spec, self.rt.ops
        o = self.rt.empty(x.shape[0], self.vv, dtype=torch.float32)
        # [T, q | k or f | v | g]
        proj = ops.linear(x, self.w_in) if self.position is None else ops.linear(x, self.w_in, out_dtype=torch.float32)
        if self.position is None:
            self._walk(proj, ctx, cache, o)
        else:
            # prompt portions in chunks on the tensor cores where they can be, the rest walked
            first = ops.chunk_scan_first(ctx, self.rt.dtype, s.key_dim, s.value_dim) if self.log_decay is not None else None
            if first is None:
                ops.turn_heads(proj, 0, self.qk, s.num_heads, s.key_dim, self.table[0], ctx)
                self._walk(proj, ctx, cache, o)
            elif first:                             # single tokens in front of the portions
                ops.turn_heads(proj, 0, self.qk, s.num_heads, s.key_dim, self.table[0], ctx, tokens=first)
                self._walk(proj, ctx, cache, o, requests=first)
            if first is not None:
                qk = self.qk
                rows = ops.turn_split(proj, 0, qk, 2 * qk, s.num_heads, s.key_dim, s.value_dim, self.table[0], ctx, first)
                ops.chunk_scan(rows, 0, 2 * qk, 4 * qk, s.num_heads, s.num_heads, s.key_dim, s.value_dim, cache.state, ctx, o,
                               first, q_lo=qk, k_lo=3 * qk, log_decay=self.log_decay, q_scale=self.k_scale)
        gate = proj[:, 2 * self.qk + self.vv:] if s.out_gate else None
        y = self.rt.empty(x.shape[0], self.vv)
        heads = 1 if s.out_norm == "all" else s.num_heads
        if self.plain_output:
            ops.rows_norm_gate(o, self.norm, heads, s.eps, gate, y)
        else:
            ops.delta_output(o, self.norm, heads, s.eps, gate, self.gate_act if gate is not None else "none", y)
        return ops.linear(y, self.w_out)
