"""A state space mixer with a scalar decay per token and head (Mamba-2's recurrence, "state space duality").

With h the layer's input [T, d], H heads of P value columns, a state of N rows, G groups of heads, K taps:

    z | x | B | C | raw = h W^T              widths H P, H P, G N, G N, H; one product
    x | B | C <- silu(conv(x | B | C) + b)   each channel's last K values, a token's own under the last of the stored taps
    dt = softplus(raw + dt_bias)             per token and head
    S   <- a S + B (dt x)^T,  a = exp(-A dt),  A = exp(A_log)    S [N, P] per head from zero; head i reads group i // (H / G)
    y   = S^T C + D x                        read from the NEW state
    y   = norm(y silu(z)) * w                the gate comes first; the norm in `norm_groups` equal runs of columns
    out = y Wo^T

The per-sequence state is S and the last K - 1 inputs of the convolution, both float32. Steps, decays, the state, what is
read from it and its norm are float32 in both engines; a bfloat16 engine rounds the projections, and for prompts also what
the convolution leaves, to bfloat16. Prompts of a bfloat16 engine run 64 tokens at a time on the tensor cores, one-token
steps in a kernel that passes over the state once, and everything else (a float32 engine, sizes that are no multiples of
8) through the scan of the other matrix states, whose stepped form is this recurrence.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..cache.cache import StateRequest
from ..kernels import ops, trace
from .base import DeferredNorm, Mixer, ParamSpec, ScaledDelta, register_mixer
from .linear import Linear, pad_rows

_DEFAULT_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D",
                  "norm": "norm", "o": "o"}
MAX_STATE, MAX_TAPS = 512, 16           # what the kernels take


class StateSpaceMixer(Mixer):
    """params: hidden, n_heads, v_dim, state, groups, norm_groups, taps, norm_eps, names (overrides of the checkpoint
    sub-names)."""

    accepts_deferred_norm = True
    adds_to_residual = True

    def __init__(self, params, runtime):
        super().__init__(params, runtime)
        p = params
        self.hidden, self.n_heads, self.v_dim = int(p["hidden"]), int(p["n_heads"]), int(p["v_dim"])
        self.state, self.groups, self.norm_groups = int(p["state"]), int(p["groups"]), int(p["norm_groups"])
        self.taps, self.eps = int(p["taps"]), float(p["norm_eps"])
        self.inner = self.n_heads * self.v_dim
        if self.n_heads % self.groups:
            raise ValueError(f"n_heads ({self.n_heads}) must be a multiple of groups ({self.groups})")
        if self.inner % self.norm_groups:
            raise ValueError(f"{self.inner} channels are not {self.norm_groups} equal runs")
        if not 0 < self.state <= MAX_STATE:
            raise ValueError(f"state ({self.state}) exceeds what the kernels take ({MAX_STATE})")
        if not 1 <= self.taps <= MAX_TAPS:
            raise ValueError(f"taps ({self.taps}) must be between 1 and {MAX_TAPS}")
        self.n_bc = self.groups * self.state
        self.channels = self.inner + 2 * self.n_bc              # what passes the convolution
        self.dt_off = self.inner + self.channels
        self.names = dict(_DEFAULT_NAMES, **(p.get("names") or {}))
        self.proj: Linear = None
        self.o: Linear = None
        self.conv_w = self.conv_bias = self.dt_bias = self.A = self.skip = self.norm_w = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d, H = self.names, self.hidden, self.n_heads
        return {n["in"]: ParamSpec((self.dt_off + H, d)),
                n["conv"]: ParamSpec((self.channels, self.taps), role="vector", init=("uniform", -0.5, 0.5)),
                n["conv_bias"]: ParamSpec((self.channels,), role="vector", init=("normal",)),
                n["dt_bias"]: ParamSpec((H,), role="vector", init=("uniform", -4.0, -1.0)),
                n["A_log"]: ParamSpec((H,), role="vector", init=("uniform", 0.0, 2.0)),
                n["D"]: ParamSpec((H,), role="vector", init=("ones",)),
                n["norm"]: ParamSpec((self.inner,), role="vector", init=("ones",)),
                n["o"]: ParamSpec((d, self.inner))}

    def load(self, tensors):
        n = self.names
        self.proj = Linear(pad_rows(tensors[n["in"]]))          # [z | x | B | C | raw steps], whole tiles of rows
        self.o = Linear(tensors[n["o"]])
        f32 = lambda k: tensors[n[k]].to(torch.float32).contiguous()                        # noqa: E731
        self.conv_w, self.conv_bias, self.dt_bias = f32("conv").t().contiguous(), f32("conv_bias"), f32("dt_bias")
        self.A, self.skip, self.norm_w = torch.exp(f32("A_log")).contiguous(), f32("D"), f32("norm")

    def weight_bytes(self) -> int:
        return self.proj.nbytes() + self.o.nbytes() + 4 * (self.channels * (self.taps + 1) + 3 * self.n_heads + self.inner)

    def cache_requests(self) -> List[object]:
        reqs = [StateRequest("S", (self.n_heads, self.state, self.v_dim))]
        if self.taps > 1:
            reqs.append(StateRequest("conv", (self.taps - 1, self.channels)))
        return reqs

    def forward(self, x, ctx, unit, owns_cache, residual=None):
        if not owns_cache:
            raise ValueError("a layer with a recurrent state of its own cannot read another layer's cache")
        T, dev = x.shape[0], self.norm_w.device
        trace.push("QKV_proj")
        if isinstance(x, DeferredNorm):
            proj = self.proj.after_norm(x)                      # one-token steps: norm and product in one kernel
            if proj is None:
                x = x.apply()
        if not isinstance(x, DeferredNorm):
            proj = self.proj(x)                                 # [T, z | x | B | C | raw steps]
        trace.pop()
        trace.push("Recurrence")
        S, conv = unit.state["S"], unit.state["conv"] if self.taps > 1 else None
        # which form runs depends on the engine and the sizes, never on what else is in the step
        tensor_cores = not ctx.decode and self.runtime.dtype == torch.bfloat16 and \
            ops.ssm_scan_supported(self.state, self.v_dim)
        xbc = torch.empty((T, self.channels), dtype=torch.bfloat16 if tensor_cores else torch.float32, device=dev)
        ops.causal_conv(proj, self.inner, None, self.conv_w, self.conv_bias, conv, ctx.cu_q, ctx.tok_seq, ctx.seq_slot, xbc,
                        act=ops.ACT_SILU, single=ctx.decode)
        if conv is not None and not ctx.decode:
            ops.conv_state_store(proj, self.inner, None, conv, ctx.cu_q, ctx.seq_slot, ctx.n_seqs)
        y = torch.empty((T, self.inner), dtype=torch.float32, device=dev)
        skip_x = skip = None
        if ctx.decode or tensor_cores:
            step = ops.ssm_step if ctx.decode else ops.ssm_scan
            step(proj, self.dt_off, self.dt_bias, self.A, self.skip, xbc, S, ctx.cu_q, ctx.seq_slot, y, ctx.n_seqs,
                 self.n_heads, self.groups, self.state, self.v_dim)
        else:
            dt = torch.empty((T, self.n_heads), dtype=torch.float32, device=dev)
            decay = torch.empty_like(dt)
            ops.ssm_steps(proj, self.dt_off, self.dt_bias, self.A, dt, decay)
            B = xbc[:, self.inner:self.inner + self.n_bc].contiguous()
            C = xbc[:, self.inner + self.n_bc:].contiguous()
            ops.matrix_scan(C, B, xbc[:, :self.inner], S, ctx.cu_q, ctx.seq_slot, y, ctx.n_seqs, self.n_heads, self.state,
                            self.v_dim, max_len=ctx.max_q_len, head_decay=decay, key_factor=dt, groups=self.groups)
            skip_x, skip = xbc[:, :self.inner], self.skip
        out = torch.empty((T, self.inner), dtype=self.runtime.dtype, device=dev)
        ops.gated_group_norm(y, proj[:, :self.inner], self.norm_w, self.eps, out, self.norm_groups, skip_x=skip_x, skip=skip)
        trace.pop()
        trace.push("Output_proj")
        done = residual is not None and self.o.add_into(out, residual)
        y = None if done else ScaledDelta([(self.o(out, out_dtype=torch.float32), 1.0)])
        trace.pop()
        return y


register_mixer("state_space", StateSpaceMixer)
