"""Norms, fused with the residual add that precedes them.

``rmsnorm``: y = w * x * (1/sqrt(mean(x^2) + eps)) with the sum of squares and
the scale in float32 (backends/simd/vec.go:72-85).  Parameters: ``size``,
``eps``, ``weight`` (tensor name) and optionally ``weight_offset`` (added to the
stored weight: 1 for a checkpoint that keeps its weights around zero).  Two such
norms of one hidden state come from one pass (`forward_pair`).

Handed a stream whose hidden state is kept in several copies
(`ResidualStream.copies`), ``rmsnorm`` norms their sum and applies a pending
update by its links on the way.

``layernorm``: y = (x - mean(x)) / sqrt(var(x) + eps) * w + b, var the mean of
the squared deviations, all in float32.  Parameters: ``size``, ``eps``,
``weight`` and ``bias`` (tensor names; ``bias`` None for a norm without one).
The reference has no such norm.  Handed a stream whose pending update has a norm of its
own to pass (`ResidualStream.pending_norm`), it norms the update, adds it and norms
the sum in one pass.
"""
from __future__ import annotations

from typing import List, Mapping, Optional

import torch

from ..kernels import ops
from ..weights.binder import WeightSpec
from .base import Norm, ResidualStream, Runtime, StepContext, register_part


@register_part("norm", "rmsnorm")
class RMSNorm(Norm):
    def __init__(self, spec):
        super().__init__(spec)
        self.size = int(self.param("size"))
        self.eps = float(self.param("eps"))
        self.weight_name = str(self.param("weight"))
        self.offset = float(self.p.get("weight_offset") or 0.0)
        self.weight: Optional[torch.Tensor] = None

    def weight_specs(self) -> List[WeightSpec]:
        return [WeightSpec(self.weight_name, (self.size,), role="vector", mean=1.0 - self.offset)]

    def load(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        w = tensors[self.weight_name]
        self.weight = rt.vector(w.to(torch.float32) + self.offset if self.offset else w)

    def forward_pair(self, stream: ResidualStream, ctx: StepContext, other: "Norm"):
        """(this norm's rows, `other`'s rows) of the same hidden state, from one pass where both are of this kind."""
        if not isinstance(other, RMSNorm) or other.eps != self.eps or stream.copies is not None:
            return self.forward(stream, ctx), other.forward(stream, ctx)
        n = stream.residual.shape[0]
        out, out2 = ctx.rt.empty(n, self.size), ctx.rt.empty(n, self.size)
        ops.add_rmsnorm(stream.residual, stream.pending, self.weight, self.eps, out, second=other.weight, out_second=out2)
        if stream.pending is not None:
            stream.image = None
        stream.pending = None
        return out, out2

    def forward(self, stream: ResidualStream, ctx: StepContext,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        n_out = rows.numel() if rows is not None else stream.residual.shape[0]
        out = ctx.rt.empty(n_out, self.size)
        if stream.copies is not None:
            # the hidden state is the sum of its copies; a pending update joins them by its links first
            mix, out_w = stream.pending_links if stream.pending is not None else (None, None)
            ops.hyper_norm(stream.copies, self.weight, self.eps, out, update=stream.pending, mix=mix, out_w=out_w, rows=rows)
            if rows is None:
                stream.pending, stream.pending_links, stream.image = None, None, None
            return out
        if stream.pending_norm is not None:
            raise ValueError("an update that passes a layer norm before it is added can only be followed by a layer norm")
        ops.add_rmsnorm(stream.residual, stream.pending, self.weight, self.eps, out, rows)
        if rows is None:
            if stream.pending is not None:
                stream.image = None
            stream.pending = None
        return out


@register_part("norm", "layernorm")
class LayerNorm(Norm):
    def __init__(self, spec):
        super().__init__(spec)
        self.size = int(self.param("size"))
        self.eps = float(self.param("eps"))
        self.weight_name = str(self.param("weight"))
        bias = self.p.get("bias")
        self.bias_name = str(bias) if bias else None
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None

    def weight_specs(self) -> List[WeightSpec]:
        specs = [WeightSpec(self.weight_name, (self.size,), role="vector", mean=1.0)]
        if self.bias_name:
            specs.append(WeightSpec(self.bias_name, (self.size,), role="vector", mean=0.0))
        return specs

    def load(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        self.weight = rt.vector(tensors[self.weight_name])
        self.bias = rt.vector(tensors[self.bias_name]) if self.bias_name else None

    def forward(self, stream: ResidualStream, ctx: StepContext,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        n_out = rows.numel() if rows is not None else stream.residual.shape[0]
        out = ctx.rt.empty(n_out, self.size)
        if stream.pending is not None and stream.pending_norm is not None:
            ops.layernorm_add_layernorm(stream.residual, stream.pending, *stream.pending_norm, self.weight, self.bias, self.eps, out, rows)
        else:
            ops.add_layernorm(stream.residual, stream.pending, self.weight, self.bias, self.eps, out, rows)
        if rows is None:
            if stream.pending is not None:
                stream.image = None
            stream.pending, stream.pending_norm = None, None
        return out
