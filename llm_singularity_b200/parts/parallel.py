"""Mixers side by side on one input.

Every branch is a mixer of any registered kind and reads the same rows.  How the results meet is
the spec's ``combine``: each branch's result RMS-normed over the model width with a weight of its
own and the mean of those taken ("normed_mean"), or the results added with fixed factors
("weighted_sum"); one kernel either way, or for the weighted sum none here where the caller forms it on its
way (``open_sum``).  In a step of few rows the branches run on streams of their own.  The branches' caches travel under one cache id as a ``CompositeCacheSpec``:
pages for the branches that keep keys and values, the request's slot row for those with state.
"""
from __future__ import annotations

from typing import Dict

from .base import MIXERS, CompositeCacheSpec, ParamSpec, Part, register_mixer
from .norm import BranchSum


@register_mixer("parallel")
class ParallelMixer(Part):
    kernels = ("sandwich",)

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        if not spec.branches or len(spec.names) != len(spec.branches) or len(set(spec.names)) != len(spec.names):
            raise ValueError("a parallel mixer needs branches, each with a name of its own")
        self.combine = getattr(spec, "combine", "normed_mean")
        if self.combine not in ("normed_mean", "weighted_sum"):
            raise ValueError(f"combine '{self.combine}' is not known (normed_mean, weighted_sum)")
        if self.combine == "weighted_sum" and len(spec.scales) != len(spec.branches):
            raise ValueError("a weighted sum needs one factor per branch")
        self.branches = [MIXERS.build(b, rt) for b in spec.branches]
        self.opens_sum = self.combine == "weighted_sum"
        self.bias = None                            # of the branches' output projections, with their factors (made at first use)
        self.graph_safe = all(getattr(b, "graph_safe", False) for b in self.branches)

    @classmethod
    def params(cls, spec) -> Dict[str, ParamSpec]:
        if getattr(spec, "combine", "normed_mean") == "weighted_sum":
            return {}
        return {f"{n}_out": ParamSpec((spec.hidden_size,), role="vector", init="ones") for n in spec.names}

    def children(self) -> Dict[str, Part]:
        return dict(zip(self.spec.names, self.branches))

    def load(self, tensors):
        self.weights = [tensors[f"{n}_out"] for n in self.spec.names] if self.combine == "normed_mean" else []

    def cache_spec(self):
        return CompositeCacheSpec(tuple(b.cache_spec() for b in self.branches))

    def _run(self, x, ctx, cache, writes_cache):
        """The branches' results: side by side on streams of their own where there are two and the step has
        few rows."""
        opens = [self.combine == "weighted_sum" and b.opens_sum for b in self.branches]
        fns = [lambda b=b, i=i: b.forward(x, ctx, cache[i], writes_cache, **({"open_sum": True} if opens[i] else {}))
               for i, b in enumerate(self.branches)]
        both = getattr(self.rt.ops, "side_by_side", None)
        if both is not None and len(fns) == 2 and self.combine == "weighted_sum":
            return list(both(x.shape[0], x.device, *fns))
        return [fn() for fn in fns]

    def forward(self, x, ctx, cache, writes_cache: bool = True, open_sum: bool = False):
        ys = self._run(x, ctx, cache, writes_cache)
        if self.combine != "weighted_sum":
            out = self.rt.empty(*ys[0].shape)
            self.rt.ops.branch_mean(ys, self.weights, self.spec.eps, out)
            return out
        terms, scales, biases = [], [], []
        for y, s in zip(ys, self.spec.scales):
            if isinstance(y, BranchSum):
                terms += y.values
                scales += [s * f for f in y.scales]
                if y.bias is not None:
                    biases.append((s, y.bias))
            else:
                terms.append(y)
                scales.append(s)
        if biases and self.bias is None:
            self.bias = sum(float(s) * b for s, b in biases).contiguous()
        if open_sum:
            return BranchSum(terms, scales, self.bias)
        out = self.rt.empty(*terms[0].shape)
        if self.bias is not None:
            self.rt.ops.branch_sum(terms, scales, out, bias=self.bias)
        else:
            self.rt.ops.branch_sum(terms, scales, out)
        return out
