"""Two mixers side by side in one layer.

``normed_pair``: factor * (rms(a(x)) w_a + rms(b(x)) w_b) for two mixers a and b
that read the same x; each output passes an RMS norm over the hidden width with a
weight of its own.  The branches keep caches and states of their own (their
requests must not share a name).  Where both can be handed their projected rows
(`input_matrix`, `input_width`, `forward_projected`), one product projects for both.
Norms, weights and the sum are float32; where a block offers its residual stream
the sum joins it in the same kernel and None is returned.

Parameters: ``hidden_size``, ``left`` and ``right`` (mixer PartSpecs),
``left_norm`` and ``right_norm`` (tensor names), ``eps``, ``factor``.  The reference
has no such mixer.
"""
from __future__ import annotations

from typing import List, Mapping, Optional

import torch

from ..cache import CacheHandle
from ..kernels import ops
from ..weights.binder import WeightSpec
from .base import Mixer, Runtime, StepContext, build_part, register_part


@register_part("mixer", "normed_pair")
class NormedPair(Mixer):
    def __init__(self, spec):
        super().__init__(spec)
        self.hidden = int(self.param("hidden_size"))
        self.branches = [build_part("mixer", self.param(name)) for name in ("left", "right")]
        self.norm_names = [str(self.param(name)) for name in ("left_norm", "right_norm")]
        self.eps = float(self.param("eps"))
        self.factor = float(self.param("factor"))
        self.shared_input = all(hasattr(b, "forward_projected") for b in self.branches)
        for b in self.branches:
            b.shares_input = self.shared_input
        self.w_in: Optional[torch.Tensor] = None
        self.norms: List[torch.Tensor] = []

    def children(self):
        return list(self.branches)

    def weight_specs(self) -> List[WeightSpec]:
        return [WeightSpec(name, (self.hidden,), role="vector", mean=1.0) for name in self.norm_names]

    def load(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        self.norms = [rt.vector(tensors[name]) for name in self.norm_names]
        if self.shared_input:
            # every branch's rows start at a multiple of 8: the products' and the kernels' 16-byte boundaries
            parts: List[torch.Tensor] = []
            self.starts = []
            at = 0
            for b in self.branches:
                self.starts.append(at)
                matrices = [m.to(rt.dtype) for m in b.input_matrix(tensors)]
                more = -b.input_width % 8
                parts += matrices + ([matrices[0].new_zeros((more, self.hidden))] if more else [])
                at += b.input_width + more
            self.w_in = rt.matrix(torch.cat(parts, dim=0))

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheHandle) -> Optional[torch.Tensor]:
        rt, n = ctx.rt, x.shape[0]
        stream, ctx.update_into = ctx.update_into, None       # the branches' updates are normed before they join anything
        try:
            if self.shared_input:
                proj = rt.empty(n, self.w_in.shape[0])
                ops.linear(x, self.w_in, proj)
                outs = [b.forward_projected(proj[:, at: at + b.input_width], x, ctx, cache) for b, at in zip(self.branches, self.starts)]
            else:
                outs = [b.forward(x, ctx, cache) for b in self.branches]
        finally:
            ctx.update_into = stream
        if stream is not None and stream.pending is None:
            ops.normed_pair(*outs, *self.norms, self.eps, self.factor, residual=stream.residual)
            stream.image = None
            return None
        out = rt.empty(n, self.hidden)
        ops.normed_pair(*outs, *self.norms, self.eps, self.factor, out=out)
        return out
