"""Mixers over a matrix state per head whose decays are per key channel, or whose writes depend on what the state holds.
What a sequence leaves behind is kept per (layer, slot) in float32 by the cache's state area and zeroed when a slot is
taken. With u [T, d] the input, H heads, D query/key channels and Dv value channels a head:

`key_decay_attention` — gated linear attention:

    q = u Wq^T D^(-1/2), k = u Wk^T, v = u Wv^T
    a = sigmoid((u Wa1^T) Wa2^T + b)^(1/tau)             a decay per head and key channel, from a low-rank product
    S_t = diag(a_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t            S [D, Dv] per head from zero
    y = (concat_h(o_h / sqrt(mean(o_h^2) + eps) * w) (.) silu(u Wg^T)) Wo^T         w [Dv] shared by the heads

`time_mixing` — RWKV's time mixing; u' is the previous token's u (zeros before the first token):

    m_s = u + (u' - u) (.) mu_s  for s in r, k, v, g, w
    r = m_r Wr^T, k = m_k Wk^T, v = m_v Wv^T, gate = silu(m_g Wg^T)
    a = exp(-exp(tanh(m_w W1^T) W2^T + w0))              a decay per head and key channel
    o_t = (S_(t-1) + diag(b) k_t v_t^T)^T r_t            read from the OLD state; b a bonus for the current token
    S_t = diag(a_t) S_(t-1) + k_t v_t^T
    y = (concat_h(o_h / sqrt(mean(o_h^2) + eps)) (.) w (.) gate) Wo^T               w per channel of all heads

`gated_delta_rule` — the delta rule with a decay per head, behind short convolutions; G heads of q and k, each shared by
H / G heads of the state:

    q, k, v <- silu(conv(u W^T))                         each channel's last K inputs, without a bias
    q <- q / sqrt(sum q^2 + unit_eps) D^(-1/2), k <- k / sqrt(sum k^2 + unit_eps)            per head
    beta = sigmoid(u Wb^T), g = exp(-exp(A_log) softplus(u Wa^T + dt_bias))                  per head of the state
    S <- g S;  w = beta (v - S^T k);  S <- S + k w^T;  o = S^T q
    y = (concat_h(o_h / sqrt(mean(o_h^2) + eps) * w) (.) silu(u Wg^T)) Wo^T         w [Dv] shared by the heads

The state of a sequence is S, and with it the previous token's u or the convolutions' last K - 1 inputs. Decays, their
logarithms and exponentials, rates, unit vectors, states and the norms of what is read are float32 in both engines; the
projections (and for prompts of a bfloat16 engine what the convolutions leave) have the activation type. One-token steps
run the recurrence with its gates, norm and output gate as one kernel; everything else goes through a scan over the piece's
tokens in order, so that a piece's arithmetic does not depend on how a sequence is cut or on what else is in the step.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..cache.cache import StateRequest
from ..kernels import ops, trace
from .base import Mixer, ParamSpec, register_mixer
from .linear import Linear, pad_rows

RANDOM_RANK = 16          # rows of a low-rank product in the random-weights mode; a checkpoint decides its own
MAX_TAPS = 16             # what the convolution kernels take


def _f32(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.float32).contiguous()


def _stack_rows(ws) -> torch.Tensor:
    dtype = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
    return torch.cat([w.to(dtype) for w in ws], dim=0)


class _MatrixState(Mixer):
    """What the three mixers share: sizes, the state request, and the scan or the one-token step."""
    form = None

    def _sizes(self, params, v_dim: int, groups: int):
        self.hidden, self.n_heads, self.dim = int(params["hidden"]), int(params["n_heads"]), int(params["dim"])
        self.v_dim, self.groups = v_dim, groups
        if self.dim > ops.MAX_CHANNEL_DIM:
            raise ValueError(f"dim ({self.dim}) exceeds what the scan kernel takes ({ops.MAX_CHANNEL_DIM})")
        if self.n_heads % groups:
            raise ValueError(f"n_heads ({self.n_heads}) must be a multiple of the {groups} heads of q and k")
        self.eps = float(params["norm_eps"])
        self.nq, self.nv = groups * self.dim, self.n_heads * v_dim
        self._step_ok = None

    def _single(self, ctx) -> bool:
        """Whether this step runs the one-token kernel."""
        if self._step_ok is None:
            self._step_ok = ops.state_step_supported(self.dim, self.v_dim)
        return ctx.decode and self._step_ok

    def _state_args(self, ctx, unit):
        return unit.state["S"], ctx.cu_q, ctx.seq_slot

    def _geometry(self, ctx):
        return ctx.n_seqs, self.n_heads, self.groups, self.dim, self.v_dim

    def _own(self, owns_cache: bool) -> None:
        if not owns_cache:
            raise ValueError("a layer with a recurrent state of its own cannot read another layer's cache")


class KeyDecayAttention(_MatrixState):
    """params: hidden, n_heads, dim, v_dim, tau, norm_eps, names (overrides of the checkpoint sub-names q, k, v, gate, a1,
    a2, a2_bias, norm, o)."""
    form = ops.FORM_KEY_DECAY

    def __init__(self, params, runtime):
        super().__init__(params, runtime)
        self._sizes(params, int(params["v_dim"]), int(params["n_heads"]))
        self.tau = float(params["tau"])
        self.names = dict({"q": "q", "k": "k", "v": "v", "gate": "g", "a1": "a1", "a2": "a2", "a2_bias": "a2.b",
                           "norm": "norm", "o": "o"}, **(params.get("names") or {}))

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d = self.names, self.hidden
        return {n["q"]: ParamSpec((self.nq, d)), n["k"]: ParamSpec((self.nq, d)), n["v"]: ParamSpec((self.nv, d)),
                n["gate"]: ParamSpec((self.nv, d)), n["a1"]: ParamSpec((-RANDOM_RANK, d)),
                n["a2"]: ParamSpec((self.nq, -RANDOM_RANK)),
                n["a2_bias"]: ParamSpec((self.nq,), role="vector", init=("uniform", -1.0, 3.0)),
                n["norm"]: ParamSpec((self.v_dim,), role="vector", init=("ones",)), n["o"]: ParamSpec((d, self.nv))}

    def load(self, tensors):
        n = self.names
        a1, a2 = tensors[n["a1"]], tensors[n["a2"]]
        self.rank = a1.shape[0]
        if a2.shape[1] != self.rank or self.rank > ops.MAX_GATE_RANK:
            raise ValueError(f"{n['a1']} {tuple(a1.shape)} and {n['a2']} {tuple(a2.shape)} do not make a product of rank "
                             f"up to {ops.MAX_GATE_RANK}")
        # [q | k | v | gate | a1], whole tiles of rows
        self.proj = Linear(pad_rows(_stack_rows([tensors[n["q"]], tensors[n["k"]], tensors[n["v"]], tensors[n["gate"]], a1])))
        self.o = Linear(tensors[n["o"]])
        self.a2t, self.a2_bias, self.norm_w = _f32(a2.t()), _f32(tensors[n["a2_bias"]]), _f32(tensors[n["norm"]])

    def weight_bytes(self) -> int:
        return self.proj.nbytes() + self.o.nbytes() + 4 * (self.a2t.numel() + self.nq + self.v_dim)

    def cache_requests(self) -> List[object]:
        return [StateRequest("S", (self.n_heads, self.dim, self.v_dim))]

    def forward(self, x, ctx, unit, owns_cache):
        self._own(owns_cache)
        T, dev, nq, nv = x.shape[0], x.device, self.nq, self.nv
        trace.push("QKV_proj")
        proj = self.proj(x)
        trace.pop()
        trace.push("Recurrence")
        q, k, v, z = proj[:, :nq], proj[:, nq:2 * nq], proj[:, 2 * nq:2 * nq + nv], proj[:, 2 * nq + nv:2 * nq + 2 * nv]
        low = proj[:, 2 * nq + 2 * nv:2 * nq + 2 * nv + self.rank]
        out = torch.empty((T, nv), dtype=proj.dtype, device=dev)
        scale = self.dim ** -0.5
        if self._single(ctx):
            ops.state_step(self.form, q, k, v, *self._state_args(ctx, unit), out, *self._geometry(ctx), self.norm_w, self.eps,
                           z, q_scale=scale, x=low, Bt=self.a2t, gate_bias=self.a2_bias, gate_mode=ops.GATE_POWER,
                           tau=self.tau)
        else:
            decay = torch.empty((T, nq), dtype=torch.float32, device=dev)
            ops.low_rank_gate(low, self.a2t, self.a2_bias, decay, ops.GATE_POWER, self.tau)
            read = torch.empty((T, nv), dtype=torch.float32, device=dev)
            ops.channel_scan(self.form, q, k, v, *self._state_args(ctx, unit), read, *self._geometry(ctx), q_scale=scale,
                             gate=decay, max_len=ctx.max_q_len)
            ops.head_rmsnorm(read, self.norm_w, self.eps, out, self.v_dim, gate=z, gate_silu=True)
        trace.pop()
        trace.push("Output_proj")
        y = self.o(out, out_dtype=torch.float32)
        trace.pop()
        return y


register_mixer("key_decay_attention", KeyDecayAttention)


class TimeMixing(_MatrixState):
    """params: hidden, n_heads, dim (of keys and of values), norm_eps, names (overrides of the checkpoint sub-names mu (a
    pattern with {s}), r, k, v, gate, w1, w2, w0, u, norm, o)."""
    form = ops.FORM_BONUS
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, params, runtime):
        super().__init__(params, runtime)
        self._sizes(params, int(params["dim"]), int(params["n_heads"]))
        self.names = dict({"mu": "mu.{s}", "r": "r", "k": "k", "v": "v", "gate": "g", "w1": "w1", "w2": "w2", "w0": "w0",
                           "u": "u", "norm": "norm", "o": "o"}, **(params.get("names") or {}))

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d = self.names, self.hidden
        vec = dict(role="vector", init=("uniform", 0.0, 1.0))
        specs = {n["mu"].format(s=s): ParamSpec((d,), **vec) for s in self.MIXES}
        specs.update({n[key]: ParamSpec((self.nq, d)) for key in ("r", "k", "v", "gate")})
        specs.update({n["w1"]: ParamSpec((-RANDOM_RANK, d)), n["w2"]: ParamSpec((self.nq, -RANDOM_RANK)),
                      n["w0"]: ParamSpec((self.nq,), role="vector", init=("uniform", -6.0, -1.0)),
                      n["u"]: ParamSpec((self.n_heads, self.dim), **vec),
                      n["norm"]: ParamSpec((self.nq,), role="vector", init=("ones",)), n["o"]: ParamSpec((d, self.nq))})
        return specs

    def load(self, tensors):
        n = self.names
        w1, w2 = tensors[n["w1"]], tensors[n["w2"]]
        self.rank = w1.shape[0]
        if w2.shape[1] != self.rank or self.rank > ops.MAX_GATE_RANK:
            raise ValueError(f"{n['w1']} {tuple(w1.shape)} and {n['w2']} {tuple(w2.shape)} do not make a product of rank "
                             f"up to {ops.MAX_GATE_RANK}")
        self.mu = _f32(torch.stack([tensors[n["mu"].format(s=s)] for s in self.MIXES]))
        ws = [tensors[n[key]] for key in ("r", "k", "v", "gate")]
        self.rkvg = _stack_rows(ws).view(4, self.nq, self.hidden).contiguous()       # four products with inputs of their own
        self.w1 = Linear(pad_rows(w1))
        self.o = Linear(tensors[n["o"]])
        self.w2t, self.w0 = _f32(w2.t()), _f32(tensors[n["w0"]])
        self.bonus, self.norm_w = _f32(tensors[n["u"]]).view(-1), _f32(tensors[n["norm"]])

    def weight_bytes(self) -> int:
        return self.rkvg.numel() * self.rkvg.element_size() + self.w1.nbytes() + self.o.nbytes() + \
            4 * (self.mu.numel() + self.w2t.numel() + 3 * self.nq)

    def cache_requests(self) -> List[object]:
        return [StateRequest("S", (self.n_heads, self.dim, self.dim)), StateRequest("previous", (1, self.hidden))]

    def forward(self, x, ctx, unit, owns_cache):
        self._own(owns_cache)
        T, dev, nq = x.shape[0], x.device, self.nq
        trace.push("QKV_proj")
        mixed = torch.empty((5, T, self.hidden), dtype=x.dtype, device=dev)
        ops.shift_mix(x, unit.state["previous"], self.mu, ctx.cu_q, ctx.tok_seq, ctx.seq_slot, mixed, single=ctx.decode)
        if not ctx.decode:
            ops.conv_state_store(x, 0, None, unit.state["previous"], ctx.cu_q, ctx.seq_slot, ctx.n_seqs)
        w = self.rkvg
        rkvg = torch.empty((4, T, nq), dtype=x.dtype, device=dev)
        if w.dtype == x.dtype:
            ops.stacked_gemm_nt(mixed[:4], w, rkvg)
        else:                                      # weights stored in 32-bit: their products run in 32-bit
            wide = torch.empty((4, T, nq), dtype=torch.float32, device=dev)
            rkvg.copy_(ops.stacked_gemm_nt(mixed[:4].to(torch.float32), w.to(torch.float32), wide))
        low = self.w1(mixed[4], out_dtype=torch.float32)[:, :self.rank]
        trace.pop()
        trace.push("Recurrence")
        r, k, v, z = rkvg[0], rkvg[1], rkvg[2], rkvg[3]
        out = torch.empty((T, nq), dtype=x.dtype, device=dev)
        if self._single(ctx):
            ops.state_step(self.form, r, k, v, *self._state_args(ctx, unit), out, *self._geometry(ctx), self.norm_w, self.eps,
                           z, bonus=self.bonus, x=low, Bt=self.w2t, gate_bias=self.w0, gate_mode=ops.GATE_DOUBLE_EXP)
        else:
            decay = torch.empty((T, nq), dtype=torch.float32, device=dev)
            ops.low_rank_gate(low, self.w2t, self.w0, decay, ops.GATE_DOUBLE_EXP)
            read = torch.empty((T, nq), dtype=torch.float32, device=dev)
            ops.channel_scan(self.form, r, k, v, *self._state_args(ctx, unit), read, *self._geometry(ctx), gate=decay,
                             bonus=self.bonus, max_len=ctx.max_q_len)
            ops.head_rmsnorm(read, self.norm_w, self.eps, out, self.dim, gate=z, gate_silu=True)
        trace.pop()
        trace.push("Output_proj")
        y = self.o(out, out_dtype=torch.float32)
        trace.pop()
        return y


register_mixer("time_mixing", TimeMixing)


class GatedDeltaRule(_MatrixState):
    """params: hidden, n_heads, n_kv_heads (heads of q and k), dim, v_dim, taps, unit_eps (under the root of the unit
    vectors), norm_eps, names (overrides of the checkpoint sub-names q, k, v, conv (a pattern with {name}), b, a, A_log,
    dt_bias, gate, norm, o)."""
    form = ops.FORM_DELTA

    def __init__(self, params, runtime):
        super().__init__(params, runtime)
        self._sizes(params, int(params["v_dim"]), int(params["n_kv_heads"]))
        self.taps, self.unit_eps = int(params["taps"]), float(params["unit_eps"])
        if not 1 <= self.taps <= MAX_TAPS:
            raise ValueError(f"taps ({self.taps}) must be between 1 and {MAX_TAPS}")
        self.channels = 2 * self.nq + self.nv
        self.names = dict({"q": "q", "k": "k", "v": "v", "conv": "{name}.conv", "b": "b", "a": "a", "A_log": "A_log",
                           "dt_bias": "dt_bias", "gate": "g", "norm": "norm", "o": "o"}, **(params.get("names") or {}))

    def _conv_name(self, which: str) -> str:
        return self.names["conv"].format(name=self.names[which])

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d, H = self.names, self.hidden, self.n_heads
        specs = {}
        for which, rows in (("q", self.nq), ("k", self.nq), ("v", self.nv)):
            specs[n[which]] = ParamSpec((rows, d))
            specs[self._conv_name(which)] = ParamSpec((rows, self.taps), role="vector", init=("uniform", -0.5, 0.5))
        specs.update({n["b"]: ParamSpec((H, d)), n["a"]: ParamSpec((H, d)),
                      n["A_log"]: ParamSpec((H,), role="vector", init=("uniform", 0.0, 2.0)),
                      n["dt_bias"]: ParamSpec((H,), role="vector", init=("uniform", -4.0, -1.0)),
                      n["gate"]: ParamSpec((self.nv, d)),
                      n["norm"]: ParamSpec((self.v_dim,), role="vector", init=("ones",)), n["o"]: ParamSpec((d, self.nv))})
        return specs

    def load(self, tensors):
        n = self.names
        # [q | k | v | gate | b | a], whole tiles of rows
        self.proj = Linear(pad_rows(_stack_rows([tensors[n[key]] for key in ("q", "k", "v", "gate", "b", "a")])))
        self.o = Linear(tensors[n["o"]])
        self.conv_w = _f32(torch.cat([_f32(tensors[self._conv_name(which)]) for which in ("q", "k", "v")]).t())    # [taps, C]
        self.A, self.dt_bias = torch.exp(_f32(tensors[n["A_log"]])).contiguous(), _f32(tensors[n["dt_bias"]])
        self.norm_w = _f32(tensors[n["norm"]])

    def weight_bytes(self) -> int:
        return self.proj.nbytes() + self.o.nbytes() + 4 * (self.channels * self.taps + 2 * self.n_heads + self.v_dim)

    def cache_requests(self) -> List[object]:
        reqs = [StateRequest("S", (self.n_heads, self.dim, self.v_dim))]
        if self.taps > 1:
            reqs.append(StateRequest("conv", (self.taps - 1, self.channels)))
        return reqs

    def forward(self, x, ctx, unit, owns_cache):
        self._own(owns_cache)
        T, dev, nq, nv, C = x.shape[0], x.device, self.nq, self.nv, self.channels
        trace.push("QKV_proj")
        proj = self.proj(x)
        trace.pop()
        trace.push("Recurrence")
        single = self._single(ctx)
        conv = unit.state["conv"] if self.taps > 1 else None
        qkv = torch.empty((T, C), dtype=torch.float32 if single else proj.dtype, device=dev)
        ops.causal_conv(proj, 0, None, self.conv_w, None, conv, ctx.cu_q, ctx.tok_seq, ctx.seq_slot, qkv, act=ops.ACT_SILU,
                        single=ctx.decode)
        if conv is not None and not ctx.decode:
            ops.conv_state_store(proj, 0, None, conv, ctx.cu_q, ctx.seq_slot, ctx.n_seqs)
        z, b_off = proj[:, C:C + nv], C + nv
        a_off, v, scale = b_off + self.n_heads, qkv[:, 2 * nq:], self.dim ** -0.5
        out = torch.empty((T, nv), dtype=proj.dtype, device=dev)
        if single:
            ops.state_step(self.form, qkv[:, :nq], qkv[:, nq:2 * nq], v, *self._state_args(ctx, unit), out,
                           *self._geometry(ctx), self.norm_w, self.eps, z, q_scale=scale, ba=proj, b_off=b_off, a_off=a_off,
                           A=self.A, dt_bias=self.dt_bias, unit_eps=self.unit_eps)
        else:
            f32 = dict(dtype=torch.float32, device=dev)
            q, k = torch.empty((T, nq), **f32), torch.empty((T, nq), **f32)
            scal, qk = torch.empty((T, self.n_heads, 2), **f32), torch.empty((T, self.groups), **f32)
            ops.delta_prepare(qkv, proj, b_off, a_off, self.A, self.dt_bias, self.unit_eps, scale, q, k, scal, qk,
                              self.n_heads, self.groups, self.dim)
            read = torch.empty((T, nv), **f32)
            ops.channel_scan(self.form, q, k, v, *self._state_args(ctx, unit), read, *self._geometry(ctx), scal=scal, qk=qk)
            ops.head_rmsnorm(read, self.norm_w, self.eps, out, self.v_dim, gate=z, gate_silu=True)
        trace.pop()
        trace.push("Output_proj")
        y = self.o(out, out_dtype=torch.float32)
        trace.pop()
        return y


register_mixer("gated_delta_rule", GatedDeltaRule)
