"""Stages between layers: what some designs do to the residual stream itself before a layer of the run order, where a
group of layers that runs several times reads the embedded tokens again at the start of every pass.

`embedding_mix`: h <- Win [h; x0], x0 being what the model's embedding stage left. The product reads both halves rounded to
the activations' type, accumulates and stores the new stream in float32. The halves lie side by side in one buffer per
step: x0's is written once, the stream's before every pass by the kernel that adds whatever the layer before has left.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import ops, trace
from .base import DeferredBranchAdd, ParamSpec, ScaledDelta, StreamStage, register_stream, single_delta
from .linear import Linear


class EmbeddingMix(StreamStage):
    """params: size (the stream's width), weight_name (the matrix's name under the stage's, default "in")."""

    def __init__(self, params, runtime):
        super().__init__(params, runtime)
        self.size = int(params["size"])
        self.weight_name = str(params.get("weight_name", "in"))
        self.proj: Linear = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {self.weight_name: ParamSpec((self.size, 2 * self.size))}

    def load(self, tensors):
        self.proj = Linear(tensors[self.weight_name])

    def weight_bytes(self) -> int:
        return self.proj.nbytes()

    @property
    def _key(self):
        return ("embedding_mix", id(self))

    def begin(self, h, ctx):
        both = torch.empty((h.shape[0], 2 * self.size), dtype=self.runtime.dtype, device=h.device)
        ops.scaled_add_rmsnorm(h, None, 0.0, None, 0.0, None, None, 0.0, both[:, self.size:])
        ctx.carry[self._key] = both

    def forward(self, h, pending, ctx):
        trace.push("Stream_in")
        both = ctx.carry[self._key]
        if isinstance(pending, DeferredBranchAdd):
            h, pending = pending.apply(), None
        if not isinstance(pending, ScaledDelta):
            pending = single_delta(pending)
            pending = ScaledDelta([(pending, 1.0)]) if pending is not None else None
        if pending is None:
            ops.scaled_add_rmsnorm(h, None, 0.0, None, 0.0, None, None, 0.0, both[:, :self.size])
        else:
            pending.add_into(h, both[:, :self.size])
        h = self.proj(both, out_dtype=torch.float32)
        ctx.carry.pop("h_act", None)
        trace.pop()
        return h, None


register_stream("embedding_mix", EmbeddingMix)
