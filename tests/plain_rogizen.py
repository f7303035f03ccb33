"""A plain, slow restatement of the Rogizen design: whole sequences, no cache, no kernels, one function per mechanism.

It shares no code with the library. `cfg` is the parsed config.json (a dict), `w` maps checkpoint names to tensors;
everything runs in the dtype of the tensors it is given (the tests use float64). Notation: T tokens, d the model
width, H heads, G key/value heads (or groups), D a head's query/key size, N the rows of a state, P its columns.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def short_conv(u, taps):
    """Per channel, token t gets the K inputs up to its own, each times its tap (taps [C, K], oldest first); what lies
    before the first of u's [T, C] rows is 0."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    y = torch.zeros_like(u)
    for j in range(K):
        y = y + padded[j:j + T] * taps[:, j]
    return y


def same_chunk_mask(T, size=None):
    """ok[i, j]: j is not after i, and both lie in the same run of `size` positions counted from position 0."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    if size is not None:
        ok = ok & (i // size == j // size)
    return ok


def rotary_table(T, rot, dtype=torch.float64):
    """cos, sin [T, dims / 2], with the frequency blend and the magnitude of YaRN when `rot["scaling"]` is there."""
    dims, base = rot["dims"], rot["base"]
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    mag = 1.0
    sc = rot.get("scaling")
    if sc is not None:
        def where(turns):
            return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo = max(math.floor(where(sc["fast"])), 0)
        hi = min(math.ceil(where(sc["slow"])), dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        f = f / sc["factor"] * ramp + f * (1.0 - ramp)
        mag = 0.1 * math.log(sc["factor"]) + 1.0
    a = torch.arange(T, dtype=torch.float64)[:, None] * f[None, :]
    return (torch.cos(a) * mag).to(dtype), (torch.sin(a) * mag).to(dtype)


def rotate_pairs(x, cos, sin, dims):
    """x [T, heads, n]: the first `dims` entries in pairs (2i, 2i+1) turned by the angle of the token's position."""
    c, s = cos[:, None, :], sin[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ----------------------------------------------------------------------------------------------- mixers
def attention(h, m, w, pre, eps):
    """Grouped-query attention inside chunks of positions, behind a short convolution of the projected q and k; the
    values are the keys as the convolution leaves them, before their norm and rotation."""
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = short_conv(h @ w[pre + "q"].T + w[pre + "q.b"], w[pre + "q.conv"]).view(T, H, D)
    k = short_conv(h @ w[pre + "k"].T + w[pre + "k.b"], w[pre + "k.conv"]).view(T, G, D)
    v = k
    q = rms(q, eps) * w[pre + "q.norm"]
    k = rms(k, eps) * w[pre + "k.norm"]
    cos, sin = rotary_table(T, m["rot"], h.dtype)
    q = rotate_pairs(q, cos, sin, m["rot"]["dims"]).transpose(0, 1)
    k = rotate_pairs(k, cos, sin, m["rot"]["dims"]).transpose(0, 1).repeat_interleave(H // G, dim=0)
    v = v.transpose(0, 1).repeat_interleave(H // G, dim=0)
    s = (q @ k.transpose(1, 2)) * m["scale"]
    size = m["mask"]["size"] if m.get("mask") is not None else None
    p = torch.softmax(s.masked_fill(~same_chunk_mask(T, size), float("-inf")), dim=-1)
    return (p @ v).transpose(0, 1).reshape(T, H * D) @ w[pre + "o"].T + w[pre + "o.b"]


def state_space(xs, B, C, dt, A, D):
    """S <- exp(A dt_t) S + B_t (dt_t x_t)^T from S = 0, then y_t = S^T C_t + D x_t. xs [T, H, P], B and C [T, G, N] (head h reads
    group h // (H / G)), dt [T, H], A and D [H]; returns y [T, H, P]."""
    T, H, P = xs.shape
    G, N = B.shape[1], B.shape[2]
    B, C = B.repeat_interleave(H // G, dim=1), C.repeat_interleave(H // G, dim=1)
    S = torch.zeros(H, N, P, dtype=xs.dtype)
    out = []
    for t in range(T):
        S = torch.exp(A * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * xs[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * xs[t])
    return torch.stack(out)


def gated_group_norm(y, z, weight, groups, eps):
    """y silu(z), each of `groups` equal runs of columns divided by its own root mean square, times the weight."""
    T, n = y.shape
    y = (y * silu(z)).view(T, groups, n // groups)
    return rms(y, eps).reshape(T, n) * weight


def mamba2(h, m, w, pre, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    p = h @ w[pre + "in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, w[pre + "conv"]) + w[pre + "conv.b"])
    xs = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = torch.nn.functional.softplus(dt + w[pre + "dt_bias"])
    y = state_space(xs, B, C, dt, -torch.exp(w[pre + "A_log"]), w[pre + "D"]).reshape(T, inner)
    return gated_group_norm(y, z, w[pre + "norm"], m["norm_groups"], eps) @ w[pre + "o"].T


def dense(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


# ----------------------------------------------------------------------------------------------- the model
MIXERS = {"attention": attention, "mamba2": mamba2}


def run_order(cfg):
    """(layer, whether a pass of the loop opens here) for every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    inside = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + inside * loop["times"] + \
        [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence. `layers_out`, a list, receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = x0
    for i, opens in run_order(cfg):
        if opens:
            x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T
        layer, pre = cfg["layers"][i], f"l{i}."
        x = x + MIXERS[layer["type"]](rms(x, eps) * w[pre + "norm1"], layer["mixer"], w, pre + "mix.", eps)
        if layer.get("mlp") is not None:
            x = x + dense(rms(x, eps) * w[pre + "norm2"], w, pre + "mlp.")
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
