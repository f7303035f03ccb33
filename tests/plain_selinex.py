"""A plain, slow restatement of the Selinex design: whole sequences, no cache, no kernels, one function per
mechanism, in the precision of the tensors it is given (the tests use float64). It shares no code with the
library; the tests compare the library with it.

Notation: x [n, d] is the residual stream of one sequence of n tokens at positions 0..n-1; `w` maps checkpoint
names to tensors; `m` is a layer's `mixer` object of config.json and `f` its `mlp` object; `p` is the prefix of a
part's tensors; c is the model's constant on every branch.

    layer:    x <- x + c * out1(mixer(in1(x)));  x <- x + c * out2(ff(in2(x)))       (the second only with a feed-forward)
    in, out:  x / sqrt(mean(x^2) + eps) * (1 + weight)
    output:   logits = E in(x), E the table the tokens were looked up in
"""
import torch


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, weight, eps):
    """The layers' norm: the stored weight is the distance from one."""
    return rms_unit(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def rotate_half(x, positions, base, dims):
    """x [n, heads, D]: entry i < dims/2 of a head is paired with entry i + dims/2; the pair turns by the angle
    position * base^(-2i/dims); entries from `dims` on pass unchanged."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = positions.to(x.dtype)[:, None] * freq[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def window_visible(n, size):
    """[n, n] booleans: query i sees key j when 0 <= i - j < size (size 0: every j <= i)."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    ok = j <= i
    if size:
        ok = ok & (i - j < size)
    return ok


def window_attention(u, w, p, m, gated):
    """Grouped-query softmax attention over a sliding window, with rotated queries and keys where `m` has a rotation,
    and with one sigmoid gate per head where `gated`."""
    n = u.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (u @ w[p + "q"].T).view(n, H, D)
    k = (u @ w[p + "k"].T).view(n, G, D)
    v = (u @ w[p + "v"].T).view(n, G, Dv)
    if m.get("rot"):
        pos = torch.arange(n)
        q = rotate_half(q, pos, m["rot"]["base"], m["rot"]["dims"])
        k = rotate_half(k, pos, m["rot"]["base"], m["rot"]["dims"])
    ok = window_visible(n, m["mask"]["size"] if m.get("mask") else 0)
    heads = []
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * m["scale"]).masked_fill(~ok, float("-inf"))
        o = torch.softmax(s, dim=-1) @ v[:, g]
        if gated:
            o = o * torch.sigmoid(u @ w[p + "g"][h])[:, None]
        heads.append(o)
    return torch.cat(heads, dim=-1) @ w[p + "o"].T


def key_decay(u, w, p, tau):
    """The gated linear attention's decay per key channel: sigmoid(z)^(1/tau), z from a low-rank product."""
    z = (u @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return torch.sigmoid(z) ** (1.0 / tau)


def gated_linear_attention(u, w, p, m, eps):
    """Per head a state S [dim, vdim] from zero: S <- diag(a_t) S + k_t v_t^T, read with q_t from the NEW state; RMS
    norm per head with one shared weight; a silu gate on the concatenated heads."""
    n = u.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q = (u @ w[p + "q"].T).view(n, H, D) * D ** -0.5
    k = (u @ w[p + "k"].T).view(n, H, D)
    v = (u @ w[p + "v"].T).view(n, H, Dv)
    a = key_decay(u, w, p, m["tau"]).view(n, H, D)
    S = torch.zeros(H, D, Dv, dtype=u.dtype)
    out = []
    for t in range(n):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    o = rms_unit(torch.stack(out), eps) * w[p + "norm"]
    return (o.reshape(n, H * Dv) * silu(u @ w[p + "g"].T)) @ w[p + "o"].T


def shifted_mix(u, mu):
    """Every token's input moved towards the previous token's by the share mu per channel (zeros before the first)."""
    before = torch.cat([torch.zeros_like(u[:1]), u[:-1]])
    return u + (before - u) * mu


def double_exp_decay(mixed, w, p):
    """RWKV's decay per key channel: exp(-exp(.)) of a low-rank product with a tanh inside."""
    return torch.exp(-torch.exp(torch.tanh(mixed @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))


def time_mixing(u, w, p, m, eps):
    """RWKV's time mixing: per head a state S [dim, dim] from zero, READ before it is updated, with a bonus for the
    current token's key: o = (S + diag(b) k v^T)^T r; then S <- diag(decay) S + k v^T."""
    n = u.shape[0]
    H, D = m["heads"], m["dim"]
    mix = {s: shifted_mix(u, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].T).view(n, H, D) for s in "rkv")
    decay = double_exp_decay(mix["w"], w, p).view(n, H, D)
    bonus = w[p + "u"]
    S = torch.zeros(H, D, D, dtype=u.dtype)
    out = []
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S + bonus[:, :, None] * kv, r[t]))
        S = decay[t][:, :, None] * S + kv
    o = rms_unit(torch.stack(out), eps).reshape(n, H * D) * w[p + "norm"]
    return (o * silu(mix["g"] @ w[p + "g"].T)) @ w[p + "o"].T


def causal_conv(x, taps):
    """x [n, c], taps [c, k]: out_t = sum_j taps[:, k-1-j] x_(t-j), zeros before the sequence."""
    n, k = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, x.shape[1], dtype=x.dtype), x])
    out = torch.zeros_like(x)
    for j in range(k):
        out = out + padded[k - 1 - j:k - 1 - j + n] * taps[:, k - 1 - j]
    return out


def unit_vector(x):
    """x over its length, with 1e-6 under the root."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(u, w, p):
    """The delta rule's decay, one per token and head."""
    return torch.exp(-torch.exp(w[p + "A_log"]) * softplus(u @ w[p + "a"].T + w[p + "dt_bias"]))


def gated_delta_rule(u, w, p, m, eps):
    """Per head a state S [dim, vdim] from zero: decay, then the difference between the value and what the state
    holds under the key is written with rate beta, then the NEW state is read."""
    n = u.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(u @ w[p + s].T, w[p + s + ".conv"])) for s in "qkv")
    q, k = unit_vector(q.view(n, G, D)) * D ** -0.5, unit_vector(k.view(n, G, D))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    v = v.view(n, H, Dv)
    beta = torch.sigmoid(u @ w[p + "b"].T)
    g = head_decay(u, w, p)
    S = torch.zeros(H, D, Dv, dtype=u.dtype)
    out = []
    for t in range(n):
        S = g[t][:, None, None] * S
        held = torch.einsum("hdv,hd->hv", S, k[t])
        S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - held))[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    o = rms_unit(torch.stack(out), eps) * w[p + "norm"]
    return (o.reshape(n, H * Dv) * silu(u @ w[p + "g"].T)) @ w[p + "o"].T


def weighted_pair(u, w, p, m, eps):
    """Gated window attention beside gated linear attention, added with a constant each."""
    return m["left_scale"] * window_attention(u, w, p + "left.", m["left"], True) + \
        m["right_scale"] * gated_linear_attention(u, w, p + "right.", m["right"], eps)


def normed_pair(u, w, p, m, eps):
    """Rotated window attention beside time mixing: half the sum of the two, each RMS-normed with a plain weight."""
    left = rms_unit(window_attention(u, w, p + "left.", m["left"], False), eps) * w[p + "left.out"]
    right = rms_unit(time_mixing(u, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


def dense_ff(u, w, p, f):
    """A clamped gate and a clamped linear part that is shifted by one."""
    g = torch.clamp(u @ w[p + "gate"].T, max=f["limit"])
    up = torch.clamp(u @ w[p + "up"].T, min=-f["limit"], max=f["limit"])
    return (g * torch.sigmoid(1.702 * g) * (up + 1.0)) @ w[p + "down"].T


def group_choice_scores(s, r):
    """[n, experts] choice scores with the experts of all but the best groups at minus infinity. A group is a run of
    neighbours, its score the sum of its two largest choice scores."""
    n, E = s.shape
    count, keep = r["groups"]["count"], r["groups"]["keep"]
    size = E // count
    by_group = s.view(n, count, size)
    score = torch.topk(by_group, min(2, size), dim=-1).values.sum(-1)
    best = torch.topk(score, keep, dim=-1).indices
    kept = torch.zeros(n, count, dtype=torch.bool).scatter_(1, best, True)
    return by_group.masked_fill(~kept[:, :, None], float("-inf")).view(n, E)


def route(u, w, p, r):
    """Sigmoid scores; score + correction chooses, first groups and then experts; the bare scores weigh, not
    normalised. Returns (chosen [n, top], weights [n, top])."""
    s = torch.sigmoid(u @ w[p + "router"].T)
    chosen = torch.topk(group_choice_scores(s + w[p + "correction"], r), r["top"], dim=-1).indices
    return chosen, torch.gather(s, 1, chosen)


def choice_margin(u, w, p, r):
    """[n]: by how much the token's choice is decided: the distance between the last group kept and the best one left
    out, and between the last expert chosen and the best one not chosen, whichever is smaller."""
    s = torch.sigmoid(u @ w[p + "router"].T) + w[p + "correction"]
    n, E = s.shape
    count, keep, top = r["groups"]["count"], r["groups"]["keep"], r["top"]
    out = torch.full((n,), float("inf"), dtype=u.dtype)
    if keep < count:
        score = torch.topk(s.view(n, count, E // count), min(2, E // count), dim=-1).values.sum(-1)
        best = torch.topk(score, keep + 1, dim=-1).values
        out = torch.minimum(out, best[:, -2] - best[:, -1])
    if keep * (E // count) > top:
        best = torch.topk(group_choice_scores(s, r), top + 1, dim=-1).values
        out = torch.minimum(out, best[:, -2] - best[:, -1])
    return out


def moe(u, w, p, f):
    chosen, weights = route(u, w, p, f["router"])
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for c in range(f["router"]["top"]):
            e = f"{p}e{int(chosen[t, c])}."
            y = (silu(u[t] @ w[e + "gate"].T) * (u[t] @ w[e + "up"].T)) @ w[e + "down"].T
            out[t] = out[t] + weights[t, c] * y
    return out


def run_order(cfg):
    """Layer indices in the order they run: the loop's layers several times in a row."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


MIXERS = {"parallel": weighted_pair, "parallel_2": normed_pair, "delta": gated_delta_rule}


def forward(w, cfg, tokens, layers_out=None, margins_out=None):
    """Logits [n, vocab] of one sequence. `layers_out`, a list, receives the stream after every layer run;
    `margins_out`, a list, the routers' choice margins [n] of every run of a layer that has a router."""
    eps, c = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        u = norm_around_one(x, w[p + "norm1"], eps)
        y = MIXERS[layer["type"]](u, w, p + "mix.", layer["mixer"], eps)
        x = x + c * norm_around_one(y, w[p + "norm1b"], eps)
        f = layer.get("mlp")
        if f is not None:
            u = norm_around_one(x, w[p + "norm2"], eps)
            if margins_out is not None and f["kind"] != "dense":
                margins_out.append(choice_margin(u, w, p + "mlp.", f["router"]))
            y = dense_ff(u, w, p + "mlp.", f) if f["kind"] == "dense" else moe(u, w, p + "mlp.", f)
            x = x + c * norm_around_one(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm_around_one(x, w["final.norm"], eps) @ w["embed"].T
