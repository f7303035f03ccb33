"""Grouped-query attention behind a short causal convolution of the projected queries and keys, whose values are the keys
themselves.

With h the layer's input [T, d], H query heads and G key heads of size D (query head i reads key head i // (H / G)), K taps:

    u = h W^T + b                            for q and for k: one product over row-concatenated weights
    y_t = c_0 u_t + c_1 u_(t-1) + .. + c_(K-1) u_(t-K+1)     per channel; inputs from before the first token count as 0;
                                             the checkpoint stores a channel's factors oldest first (K = 1: one factor)
    v = y                                    of the key heads: there is no value projection
    q, k <- y / sqrt(mean_head(y^2) + eps) * w   RMS norm per head, one weight [D] for all q heads and one for all k heads
    q, k <- rotated: entries (2i, 2i + 1) of the first `rot_dims` of a head by the position's angle (YaRN's frequencies and
            magnitude when `rot_scaling` is given)
    p_ij = softmax_j(scale * q_i . k_j)      over the j <= i that i may see: all of them, the last `window`, or those of
                                             i's own chunk of `chunk` positions, chunks counted from position 0
    y = (p v) Wo^T + bo

Keys are cached normed and rotated, values as the convolution leaves them. The last K - 1 inputs u of q and k are a
per-sequence state beside the cache. Convolution, norms, rotation, scores and softmax are float32.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..cache.cache import KVRequest, StateRequest
from ..kernels import ops, trace
from .base import AttentionOptions, DeferredNorm, Mixer, ParamSpec, ScaledDelta, register_mixer
from .latent_attention import rotation_table
from .linear import Linear, pad_rows

_DEFAULT_NAMES = {"q": "q", "q_bias": "q.b", "k": "k", "k_bias": "k.b", "q_norm": "q.norm", "k_norm": "k.norm",
                  "q_conv": "q.conv", "k_conv": "k.conv", "o": "o", "o_bias": "o.b"}
MAX_HEAD_DIM, MAX_TAPS = 256, 16        # what the kernels take


class ConvAttention(Mixer):
    """params: hidden, n_heads, n_kv_heads, head_dim, taps, scale, norm_eps, rot_dims, rot_base, rot_scaling (None or
    {factor, original, fast, slow}), window (0 = none), chunk (0 = none), bias (bool: of the q, k and output projections,
    default True), names (overrides of the checkpoint sub-names)."""

    accepts_deferred_norm = True
    adds_to_residual = True

    def __init__(self, params, runtime):
        super().__init__(params, runtime)
        p = params
        self.hidden, self.n_heads, self.n_kv_heads = int(p["hidden"]), int(p["n_heads"]), int(p["n_kv_heads"])
        self.head_dim, self.taps = int(p["head_dim"]), int(p["taps"])
        if self.n_heads % self.n_kv_heads:
            raise ValueError(f"n_heads ({self.n_heads}) must be a multiple of n_kv_heads ({self.n_kv_heads})")
        if not 0 < self.head_dim <= MAX_HEAD_DIM:
            raise ValueError(f"head size {self.head_dim} exceeds what the kernels take ({MAX_HEAD_DIM})")
        if not 1 <= self.taps <= MAX_TAPS:
            raise ValueError(f"taps ({self.taps}) must be between 1 and {MAX_TAPS}")
        self.eps = float(p["norm_eps"])
        self.rot_dims = int(p["rot_dims"])
        if self.rot_dims % 2 or not 0 < self.rot_dims <= self.head_dim:
            raise ValueError(f"rot_dims ({self.rot_dims}) must be even, positive and at most head_dim ({self.head_dim})")
        self.window, self.chunk = int(p.get("window") or 0), int(p.get("chunk") or 0)
        if self.window and self.chunk:
            raise ValueError("a window or chunks, not both")
        self.options = AttentionOptions(scale=float(p["scale"]), window=self.window, chunk=self.chunk)
        self.bias = bool(p.get("bias", True))
        self.names = dict(_DEFAULT_NAMES, **(p.get("names") or {}))
        self.nq, self.nk = self.n_heads * self.head_dim, self.n_kv_heads * self.head_dim
        self.table = rotation_table(self.rot_dims, float(p["rot_base"]), runtime.max_positions, runtime.device,
                                    p.get("rot_scaling")) if runtime.device.type == "cuda" else None
        self.proj: Linear = None
        self.o: Linear = None
        self.qk_bias = self.o_bias = self.conv_w = self.q_w = self.k_w = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d, D, K = self.names, self.hidden, self.head_dim, self.taps
        vec = dict(role="vector", init=("normal",))
        specs = {n["q"]: ParamSpec((self.nq, d)), n["k"]: ParamSpec((self.nk, d)), n["o"]: ParamSpec((d, self.nq)),
                 n["q_norm"]: ParamSpec((D,), role="vector", init=("ones",)),
                 n["k_norm"]: ParamSpec((D,), role="vector", init=("ones",)),
                 n["q_conv"]: ParamSpec((self.nq, K), role="vector", init=("uniform", -0.5, 0.5)),
                 n["k_conv"]: ParamSpec((self.nk, K), role="vector", init=("uniform", -0.5, 0.5))}
        if self.bias:
            specs.update({n["q_bias"]: ParamSpec((self.nq,), **vec), n["k_bias"]: ParamSpec((self.nk,), **vec),
                          n["o_bias"]: ParamSpec((d,), **vec)})
        return specs

    def load(self, tensors):
        n = self.names
        ws = [tensors[n["q"]], tensors[n["k"]]]
        dtype = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
        self.proj = Linear(pad_rows(torch.cat([w.to(dtype) for w in ws], dim=0)))          # [q | k], whole tiles of rows
        self.o = Linear(tensors[n["o"]])
        f32 = lambda *names: torch.cat([tensors[n[k]].to(torch.float32) for k in names]).contiguous()     # noqa: E731
        self.conv_w = f32("q_conv", "k_conv").t().contiguous()                             # taps [K, C]
        self.q_w, self.k_w = f32("q_norm"), f32("k_norm")
        if self.bias:
            self.qk_bias, self.o_bias = f32("q_bias", "k_bias"), f32("o_bias")

    def weight_bytes(self) -> int:
        return self.proj.nbytes() + self.o.nbytes() + 4 * ((self.nq + self.nk) * (self.taps + 1) + self.hidden)

    def cache_requests(self) -> List[object]:
        reqs = [KVRequest(self.n_kv_heads, self.head_dim, self.window, chunk=self.chunk)]
        if self.taps > 1:
            reqs.append(StateRequest("conv", (self.taps - 1, self.nq + self.nk)))
        return reqs

    def forward(self, x, ctx, unit, owns_cache, residual=None):
        if not owns_cache:
            raise ValueError("a layer with a convolution state of its own cannot read another layer's cache")
        kv, T = unit.kv, x.shape[0]
        state = unit.state["conv"] if self.taps > 1 else None
        trace.push("QKV_proj")
        if isinstance(x, DeferredNorm):
            proj = self.proj.after_norm(x)                    # one-token steps: norm and product in one kernel
            if proj is None:
                x = x.apply()
        if not isinstance(x, DeferredNorm):
            proj = self.proj(x)                               # [T, q | k]
        trace.pop()
        trace.push("Conv+QKnorm+KV_cache")
        q = torch.empty((T, self.nq), dtype=kv.k.dtype, device=proj.device)
        ops.conv_qk_store(proj, self.qk_bias, self.conv_w, state, self.q_w, self.k_w, self.eps, self.table, self.rot_dims,
                          ctx.cu_q, ctx.tok_pos, ctx.tok_seq, ctx.seq_slot, kv.block_table, kv.page_size, q, kv.k, kv.v,
                          self.n_heads, self.n_kv_heads, self.head_dim, single=ctx.decode)
        if state is not None and not ctx.decode:
            ops.conv_state_store(proj, 0, self.qk_bias, state, ctx.cu_q, ctx.seq_slot, ctx.n_seqs)
        trace.pop()
        out = torch.empty((T, self.nq), dtype=q.dtype, device=q.device)
        trace.push("FlashDecode" if ctx.decode else "FlashAttn")
        ctx.attention(q, kv, out, self.n_heads, self.n_kv_heads, self.head_dim, self.options)
        trace.pop()
        trace.push("Output_proj")
        done = residual is not None and self.o.add_into(out, residual, self.o_bias)
        y = None if done else ScaledDelta([(self.o(out, out_dtype=torch.float32), 1.0)], bias=self.o_bias)
        trace.pop()
        return y


register_mixer("conv_attention", ConvAttention)
